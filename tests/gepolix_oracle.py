"""Plain float64 restatement of the Gepolix family, one function per mechanism, token by token where the mechanism is sequential.
Shares no code with the engine: the tests compare the engine's kernels and whole models against these functions.

Tensor names follow the family's checkpoints (`l<i>.norm1`, `l<i>.mix.*`, `l<i>.mlp.*`, `embed`, `final.norm`, `head`); a model is a
(config dict, {name: tensor}) pair."""
import torch

F64 = torch.float64


def tanh_norm(x, w, alpha, b):
    """The family's "norm" looks at no other entry of the row: squash alpha x into (-1, 1), scale and shift it."""
    return torch.tanh(x.to(F64) * float(alpha)) * w.to(F64) + b.to(F64)


def grouped_rms(x, w, groups, eps):
    """x [..., D] in `groups` consecutive parts, each over its own sqrt(mean(part^2) + eps); the whole times w."""
    parts = x.to(F64).reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    parts = parts / torch.sqrt((parts * parts).mean(-1, keepdim=True) + eps)
    return parts.reshape(x.shape) * w.to(F64)


def rotate(x, pos, dims, base):
    """x [T, heads, d]; entries i and i + dims / 2 (i < dims / 2) turn by pos base^(-2 i / dims); entries from dims on stay."""
    half = dims // 2
    ang = pos.to(F64)[:, None] * torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(half)], dtype=F64)[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], dim=-1)


def window_attention(q, k, v, scale, window, pos0=0):
    """q [T, H, d] at positions pos0 ..; k [N, G, d], v [N, G, dv] at positions 0 .. N - 1.  Query i sees j with 0 <= i - j < window
    (window 0: every j <= i); softmax over what it sees."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        i = pos0 + t
        lo = max(0, i - window + 1) if window else 0
        for hh in range(H):
            g = hh // (H // G)
            p = torch.softmax((k[lo:i + 1, g].to(F64) @ q[t, hh].to(F64)) * scale, 0)
            out[t, hh] = p @ v[lo:i + 1, g].to(F64)
    return out


def project(h, W, name):
    y = h.to(F64) @ W[name].to(F64).T
    return y + W[name + ".b"].to(F64) if name + ".b" in W else y


def attention_mixer(h, W, m, pos0=0, past=None, foreign=None):
    """h [T, D] of ONE sequence whose first row sits at pos0; past = this layer's (keys, values) of earlier positions or None; foreign = (keys,
    values) of another layer up to and including the new positions (a layer without keys and values of its own).  Returns (output [T, D],
    (keys, values))."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(pos0, pos0 + T)
    rot = m.get("rot")

    def turned(x):
        return rotate(x, pos, int(rot["dims"]), float(rot["base"])) if rot and rot.get("dims") else x

    q = turned(project(h, W, "q").reshape(T, H, d))
    if foreign is not None:
        k, v = foreign
    else:
        k, v = turned(project(h, W, "k").reshape(T, G, d)), project(h, W, "v").reshape(T, G, dv)
        if past is not None:
            k, v = torch.cat([past[0], k]), torch.cat([past[1], v])
    o = window_attention(q, k, v, float(m["scale"]), int((m.get("mask") or {}).get("size", 0)), pos0)
    return o.reshape(T, H * dv) @ W["o"].to(F64).T, (k, v)


def causal_conv_silu(u, w, b, tail=None):
    """u [T, C]; y_t = silu(b + sum_j w[:, j] u_(t - taps + 1 + j)).  tail [taps - 1, C]: the rows before the first (zeros at the start).
    Returns (y, the new tail)."""
    taps = w.shape[1]
    full = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=F64) if tail is None else tail, u.to(F64)])
    y = torch.stack([(full[t:t + taps] * w.to(F64).T).sum(0) + b.to(F64) for t in range(u.shape[0])])
    return torch.nn.functional.silu(y), full[full.shape[0] - (taps - 1):]


def ssd_recurrence(x, B, C, dt, A_log, D, S):
    """x [T, H, P], B and C [T, G, N], dt [T, H] (after softplus), S [H, N, P].  Returns (y [T, H, P], S after the last token)."""
    T, H, P = x.shape
    per = H // B.shape[1]
    y = torch.zeros(T, H, P, dtype=F64)
    S = S.clone()
    for t in range(T):
        for hh in range(H):
            g = hh // per
            S[hh] = torch.exp(-torch.exp(A_log[hh].to(F64)) * dt[t, hh]) * S[hh] + dt[t, hh] * torch.outer(B[t, g], x[t, hh])
            y[t, hh] = C[t, g] @ S[hh] + D[hh].to(F64) * x[t, hh]
    return y, S


def mamba2_mixer(h, W, m, eps, state=None):
    """h [T, D] of ONE sequence; state = (convolution tail, S) or None.  Returns (output [T, D], state)."""
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner, bc = H * P, G * N
    u = h.to(F64) @ W["in"].to(F64).T
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * bc], u[:, 2 * inner + 2 * bc:]
    tail, S = state if state is not None else (None, torch.zeros(H, N, P, dtype=F64))
    y, tail = causal_conv_silu(xbc, W["conv"], W["conv.b"], tail)
    dt = torch.nn.functional.softplus(dt + W["dt_bias"].to(F64), threshold=1e9)
    o, S = ssd_recurrence(y[:, :inner].reshape(T, H, P), y[:, inner:inner + bc].reshape(T, G, N), y[:, inner + bc:].reshape(T, G, N), dt, W["A_log"],
                          W["D"], S)
    o = grouped_rms(o.reshape(T, inner) * torch.nn.functional.silu(z), W["norm"], m["norm_groups"], eps)
    return o @ W["o"].to(F64).T, (tail, S)


def silu_ff(h, W):
    h = h.to(F64)
    return (torch.nn.functional.silu(h @ W["gate"].to(F64).T) * (h @ W["up"].to(F64).T)) @ W["down"].to(F64).T


def route(h, W, top):
    """(chosen experts [T, top], their weights): the largest biased logits, softmax over the chosen ones alone."""
    z = h.to(F64) @ W["router"].to(F64).T + W["router.b"].to(F64)
    best = z.topk(top, dim=-1)
    return best.indices, torch.softmax(best.values, -1)


def moe_ff(h, W, f):
    idx, w = route(h, W, int(f["router"]["top"]))
    h64 = h.to(F64)
    out = torch.zeros_like(h64)
    for t in range(h.shape[0]):
        for j in range(idx.shape[1]):
            e = int(idx[t, j])
            out[t] += w[t, j] * silu_ff(h64[t:t + 1], {n: W[f"e{e}.{n}"] for n in ("gate", "up", "down")})[0]
    if f.get("shared"):
        gate = torch.sigmoid(h64 @ W["shared.sg"].to(F64).T)
        out += gate * silu_ff(h64, {n: W[f"shared.{n}"] for n in ("gate", "up", "down")})
    return out


def sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def norm_of(x, weights, name):
    return tanh_norm(x, weights[name], weights[name + ".alpha"], weights[name + ".b"])


def forward(config, weights, tokens, carry=None, hook=None):
    """One sequence's next tokens; carry = per-layer state of the earlier tokens (None at the start).  Returns (logits [T, vocab], carry)."""
    eps = float(config["norm"]["eps"])
    carry = carry or {"pos": 0, "layers": [None] * len(config["layers"])}
    pos0 = carry["pos"]
    x = weights["embed"].to(F64)[torch.as_tensor(tokens, dtype=torch.long)]
    new = []
    for i, L in enumerate(config["layers"]):
        h = norm_of(x, weights, f"l{i}.norm1")
        Wm, m = sub(weights, f"l{i}.mix."), L["mixer"]
        if L["type"] == "attention":
            src = m.get("kv_from")
            y, st = attention_mixer(h, Wm, m, pos0, carry["layers"][i], None if src is None else new[src])
        elif L["type"] == "mamba2":
            y, st = mamba2_mixer(h, Wm, m, eps, carry["layers"][i])
        else:
            raise ValueError(L["type"])
        new.append(st)
        f = L.get("mlp")
        if f is not None:
            Wf = sub(weights, f"l{i}.mlp.")
            y = y + (silu_ff(h, Wf) if f["kind"] == "dense" else moe_ff(h, Wf, f))
        x = x + y
        if hook is not None:
            hook(i, x)
    return norm_of(x, weights, "final.norm") @ weights["head"].to(F64).T, {"pos": pos0 + len(tokens), "layers": new}


# ------------------------------------------------------------------------------------------------ small models for the tests
def attention_layer(heads, kv_heads, dim, vdim, window, scale=None, rot_dims=0, base=10000.0, mlp=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5}
    if window:
        m["mask"] = {"size": window}
    if rot_dims:
        m["rot"] = {"dims": rot_dims, "base": base}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def mamba2_layer(heads, vdim, state, groups=1, conv=4, norm_groups=1, mlp=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared_ff=0):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared_ff:
        f["shared"] = {"ff": shared_ff}
    return f


def make_config(layers, vocab=64, width=32, eps=1e-5):
    return {"architecture": "Gepolix", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def random_weights(cfg, seed=0, router_gain=4.0):
    """bf16 tensors under the family's names.  Projections ~ N(0, 1 / fan_in) so that activations stay O(1); decay rates and step sizes spread
    so that heads that forget at once and heads that hardly forget both occur; router rows scaled up so that selections are decided."""
    g = torch.Generator().manual_seed(seed)
    D = cfg["width"]

    def lin(o, i, gain=1.0):
        return (torch.randn(o, i, generator=g) * gain * i ** -0.5).bfloat16()

    def vec(n, mean=0.0, std=0.2):
        return (mean + std * torch.randn(n, generator=g)).bfloat16()

    w = {"embed": torch.randn(cfg["vocab"], D, generator=g).bfloat16(), "head": lin(cfg["vocab"], D, 2.0)}

    def norm(name):
        w[name], w[name + ".b"], w[name + ".alpha"] = vec(D, 1.0), vec(D), torch.tensor(0.6 + 0.3 * float(torch.rand(1, generator=g))).bfloat16()

    norm("final.norm")
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}."
        norm(p + "norm1")
        if L["type"] == "attention":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            w.update({p + "mix.q": lin(H * d, D, 1.5), p + "mix.q.b": vec(H * d, 0.0, 0.5), p + "mix.o": lin(D, H * dv)})
            if m.get("kv_from") is None:
                w.update({p + "mix.k": lin(G * d, D, 1.5), p + "mix.k.b": vec(G * d, 0.0, 0.5), p + "mix.v": lin(G * dv, D), p + "mix.v.b": vec(G * dv, 0.0, 0.5)})
        else:
            H, P, N, G, taps = m["heads"], m["vdim"], m["state"], m["groups"], m["conv"]
            inner, C = H * P, H * P + 2 * G * N
            w.update({p + "mix.in": lin(2 * inner + 2 * G * N + H, D), p + "mix.conv": lin(C, taps, 1.2), p + "mix.conv.b": vec(C), p + "mix.D": vec(H, 1.0, 0.5),
                      p + "mix.dt_bias": vec(H, -1.0, 1.0), p + "mix.A_log": vec(H, 0.0, 1.5), p + "mix.norm": vec(inner, 1.0), p + "mix.o": lin(D, inner)})
        f = L.get("mlp")
        if f is None:
            continue
        if f["kind"] == "dense":
            w.update({p + "mlp.gate": lin(f["ff"], D, 2.0), p + "mlp.up": lin(f["ff"], D, 2.0), p + "mlp.down": lin(D, f["ff"])})
            continue
        E, ff = f["router"]["experts"], f["expert"]["ff"]
        w[p + "mlp.router"], w[p + "mlp.router.b"] = lin(E, D, router_gain), vec(E, 0.0, 1.0)
        for e in range(E):
            w.update({p + f"mlp.e{e}.gate": lin(ff, D), p + f"mlp.e{e}.up": lin(ff, D), p + f"mlp.e{e}.down": lin(D, ff)})
        if f.get("shared"):
            sf = f["shared"]["ff"]
            w.update({p + "mlp.shared.gate": lin(sf, D, 1.5), p + "mlp.shared.up": lin(sf, D, 1.5), p + "mlp.shared.down": lin(D, sf), p + "mlp.shared.sg": lin(1, D, 2.0)})
    return w


def run(cfg, w, tokens, collect_layers=False):
    """Logits of every position of one sequence (float64 [T, vocab]); with collect_layers also the residual after every layer."""
    res = []
    logits, _ = forward(cfg, w, tokens, hook=(lambda i, x: res.append(x.clone())) if collect_layers else None)
    return (logits, res) if collect_layers else logits


def greedy(cfg, w, prompt, n_new):
    """Greedy continuation, recomputing the whole sequence for every new token."""
    toks, out = list(prompt), []
    for _ in range(n_new):
        nxt = int(run(cfg, w, toks)[-1].argmax())
        out.append(nxt)
        toks.append(nxt)
    return out


def write_model(folder, cfg, w):
    """config.json + model.safetensors (8-byte little-endian header length, JSON header, raw little-endian data) -> folder."""
    import json
    import os
    import struct
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as fh:
        json.dump(cfg, fh)
    names = {torch.bfloat16: "BF16", torch.float32: "F32", torch.int32: "I32"}
    header, blobs, at = {}, [], 0
    for k, t in w.items():
        raw = t.contiguous().reshape(-1).view(torch.uint8).numpy().tobytes() if t.numel() else b""
        header[k] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    hj = json.dumps(header).encode()
    hj += b" " * (-len(hj) % 8)
    with open(os.path.join(folder, "model.safetensors"), "wb") as fh:
        fh.write(struct.pack("<Q", len(hj)) + hj + b"".join(blobs))
    return folder
