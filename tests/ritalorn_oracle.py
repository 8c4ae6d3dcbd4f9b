"""Plain float64 restatement of the Ritalorn family, one function per mechanism.  Shares no code with the engine: the tests compare the engine's
kernels and whole models against these functions.

Tensor names follow the family's checkpoints (`l<i>.{norm1, ls1, hc1.*, norm2, ls2, hc2.*}`, `l<i>.mix.*`, `l<i>.mlp.*`, `embed`, `final.norm`,
`head`); a model is a (config dict, {name: tensor}) pair."""
import math

import torch

F64 = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def linear(h, W, name):
    y = h.to(F64) @ W[name].to(F64).T
    return y + W[name + ".b"].to(F64) if name + ".b" in W else y


def causal_conv(u, w, tail=None):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j).  tail [taps - 1, C]: the rows in front of the first (zeros at the start of a
    sequence).  Returns (y, the new tail)."""
    taps = w.shape[1]
    full = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=F64) if tail is None else tail, u])
    y = sum(full[j:j + u.shape[0]] * w[:, j].to(F64) for j in range(taps))
    return y, full[full.shape[0] - (taps - 1):]


def rotate_pairs(x, pos, dims, base):
    """x [T, ..., n]; entries 2i and 2i + 1 (2i < dims) turn by pos base^(-2i / dims); entries from dims on stay."""
    out = x.clone()
    for i in range(dims // 2):
        a = pos.to(F64) * float(base) ** (-2.0 * i / dims)
        a = a.reshape(-1, *([1] * (x.dim() - 2)))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a)
    return out


def linear_slopes(H):
    """Heads lose 2^(-8 / H), 2^(-16 / H), .., 2^-8 of a score per position of distance."""
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)], dtype=F64)


def sees_window(i, j, size):
    return (j <= i) & (i - j < size) if size else j <= i


def sees_part(i, j, size):
    return (j <= i) & (i // size == j // size) if size else j <= i


def attend(q, k, v, scale, sees, pos0=0, slopes=None):
    """q [T, H, d] at positions pos0 ..; k [N, G, d], v [N, G, dv] at positions 0 .. N - 1; sees(i, j): whether query i sees key j (tensors of
    positions);
    slopes [H]: what a score loses per position of distance.  Softmax over what a query sees -> [T, H, dv]."""
    T, H, _ = q.shape
    N, G, _ = k.shape
    per = H // G
    i, j = torch.arange(pos0, pos0 + T)[:, None], torch.arange(N)[None, :]
    seen = sees(i, j)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T) * scale
        if slopes is not None:
            s = s - slopes[h] * (i - j).to(F64)
        out[:, h] = torch.softmax(s.masked_fill(~seen, -math.inf), -1) @ v[:, h // per]
    return out


def attention_mixer(h, W, m, eps, pos0=0, past=None, foreign=None):
    """h [T, D] of ONE sequence whose first row sits at pos0.  past = (this layer's convolution tails by name, keys, values) or None; foreign =
    (keys, values) of another layer up to and including the new positions (a layer without keys and values of its own).  Returns (output [T, D],
    (tails, keys, values))."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    tails = {}

    def projected(name):
        u = linear(h, W, name)
        if name + ".conv" in W:
            u, tails[name] = causal_conv(u, W[name + ".conv"], past[0][name] if past is not None else None)
        return u

    q = rms(projected("q").reshape(T, H, d), eps)
    if foreign is not None:
        k, v = foreign
    else:
        k, v = rms(projected("k").reshape(T, G, d), eps), projected("v").reshape(T, G, dv)
        if past is not None:
            k, v = torch.cat([past[1], k]), torch.cat([past[2], v])
    size = int((m.get("mask") or {}).get("size", 0))
    o = attend(q, k, v, float(m["scale"]), lambda i, j: sees_part(i, j, size), pos0, linear_slopes(H)).reshape(T, H * dv)
    return linear(o * torch.sigmoid(linear(h, W, "g")), W, "o"), (tails, k, v)


def latent_mixer(h, W, m, eps, pos0=0, past=None):
    """h [T, D] of ONE sequence; past = the (latents, rotated key parts) of earlier positions or None.  Every head's keys and values are formed
    explicitly.  Returns (output [T, D], (latents, rotated parts))."""
    T = h.shape[0]
    H, d, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    rot = m.get("rot") or {}
    pos = torch.arange(pos0, pos0 + T)
    dims, base = int(rot.get("dims", dr)), float(rot.get("base", 10000.0))
    q = linear(h, W, "q").reshape(T, H, d + dr)
    q = torch.cat([q[..., :d], rotate_pairs(q[..., d:], pos, dims, base)], -1)
    low = linear(h, W, "dkv")
    c, kr = rms(low[:, :R], eps) * W["dkv.norm"].to(F64), rotate_pairs(low[:, R:], pos, dims, base)
    if past is not None:
        c, kr = torch.cat([past[0], c]), torch.cat([past[1], kr])
    N = c.shape[0]
    k = torch.cat([linear(c, W, "uk").reshape(N, H, d), kr[:, None, :].expand(N, H, dr)], -1)
    v = linear(c, W, "uv").reshape(N, H, dv)
    size = int((m.get("mask") or {}).get("size", 0))
    o = attend(q, k, v, float(m["scale"]), lambda i, j: sees_window(i, j, size), pos0)
    return linear(o.reshape(T, H * dv), W, "o"), (c, kr)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gated_ff(h, W):
    return linear(gelu_tanh(linear(h, W, "gate")) * linear(h, W, "up"), W, "down")


def read_streams(X, w_in):
    """X [streams, T, D] -> the weighted sum a sublayer's norm reads."""
    return sum(float(w_in[s]) * X[s] for s in range(X.shape[0]))


def write_streams(X, mix, w_out, y):
    """All streams at once from the old ones: stream t becomes sum_s mix[s, t] X_s + w_out[t] y."""
    S = X.shape[0]
    return torch.stack([sum(float(mix[s, t]) * X[s] for s in range(S)) + float(w_out[t]) * y for t in range(S)])


def sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(config, weights, tokens, carry=None, hook=None):
    """One sequence's next tokens; carry = per-layer state of the earlier tokens (None at the start).  Returns (logits [T, vocab], carry)."""
    eps = float(config["norm"]["eps"])
    carry = carry or {"pos": 0, "layers": [None] * len(config["layers"])}
    pos0, n = carry["pos"], int(config.get("streams", 1))
    e = weights["embed"].to(F64)[torch.as_tensor(tokens, dtype=torch.long)]
    X = torch.stack([e] * n)
    new = []
    for i, L in enumerate(config["layers"]):
        p, m = f"l{i}.", L["mixer"]

        def sublayer(X, q, fn):
            u = read_streams(X, weights[p + f"hc{q}.in"].to(F64))
            y = fn(rms(u, eps) * weights[p + f"norm{q}"].to(F64)) * weights[p + f"ls{q}"].to(F64)
            return write_streams(X, weights[p + f"hc{q}.mix"].to(F64), weights[p + f"hc{q}.out"].to(F64), y)

        def mixer(h):
            W = sub(weights, p + "mix.")
            if L["type"] == "attention":
                src = m.get("kv_from")
                y, st = attention_mixer(h, W, m, eps, pos0, carry["layers"][i], None if src is None else new[src][1:])
            elif L["type"] == "latent_attention":
                y, st = latent_mixer(h, W, m, eps, pos0, carry["layers"][i])
            else:
                raise ValueError(L["type"])
            new.append(st)
            return y

        X = sublayer(X, 1, mixer)
        if L.get("mlp") is not None:
            X = sublayer(X, 2, lambda h: gated_ff(h, sub(weights, p + "mlp.")))
        if hook is not None:
            hook(i, X.sum(0))
    logits = linear(rms(X.sum(0), eps) * weights["final.norm"].to(F64), weights, "head")
    cap = float(config.get("logit_softcap", 0.0))
    return (cap * torch.tanh(logits / cap) if cap else logits), {"pos": pos0 + len(tokens), "layers": new}


# ------------------------------------------------------------------------------------------------ small models for the tests
def attention_layer(heads, kv_heads, dim, vdim, chunk, scale=None, conv=3, ff=0, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5}
    if conv:
        m["conv"] = conv
    if chunk:
        m["mask"] = {"size": chunk}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent_layer(heads, dim, rot_dim, vdim, kv_rank, window, scale=None, base=10000.0, ff=0):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale if scale is not None else (dim + rot_dim) ** -0.5,
         "rot": {"dims": rot_dim, "base": base}}
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def make_config(layers, vocab=64, width=32, eps=1e-5, streams=3, softcap=9.0):
    return {"architecture": "Ritalorn", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "streams": streams, "logit_softcap": softcap}


def random_weights(cfg, seed=0):
    """bf16 tensors under the family's names.  Projections ~ N(0, 1 / fan_in) so that activations stay O(1); mixing matrices that are neither
    symmetric nor close to the identity; layer scales and stream weights that differ from entry to entry."""
    g = torch.Generator().manual_seed(seed)
    D, S = cfg["width"], cfg["streams"]

    def lin(o, i, gain=1.0):
        return (torch.randn(o, i, generator=g) * gain * i ** -0.5).bfloat16()

    def vec(n, mean=0.0, std=0.2):
        return (mean + std * torch.randn(n, generator=g)).bfloat16()

    w = {"embed": torch.randn(cfg["vocab"], D, generator=g).bfloat16(), "head": lin(cfg["vocab"], D, 3.0), "final.norm": vec(D, 1.0)}

    def sublayer(p, q):
        w.update({p + f"norm{q}": vec(D, 1.0), p + f"ls{q}": vec(D, 0.7, 0.3), p + f"hc{q}.in": vec(S, 1.0 / S, 0.4), p + f"hc{q}.out": vec(S, 1.0, 0.4),
                  p + f"hc{q}.mix": (0.8 * torch.eye(S) + 0.3 * torch.randn(S, S, generator=g)).bfloat16()})

    for i, L in enumerate(cfg["layers"]):
        m, p, a = L["mixer"], f"l{i}.", f"l{i}.mix."
        sublayer(p, 1)
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        if L["type"] == "attention":
            G = m["kv_heads"]
            for name, n in (("q", H * d), ("k", G * d), ("v", G * dv)) if m.get("kv_from") is None else (("q", H * d), ):
                w.update({a + name: lin(n, D), a + name + ".b": vec(n, 0.0, 0.4)})
                if m.get("conv"):
                    w[a + name + ".conv"] = vec((n, m["conv"]), 0.0, 0.8)
            w.update({a + "g": lin(H * dv, D, 2.0), a + "o": lin(D, H * dv, 2.0), a + "o.b": vec(D)})
        else:
            dr, R = m["rot_dim"], m["kv_rank"]
            w.update({a + "q": lin(H * (d + dr), D, 1.5), a + "dkv": lin(R + dr, D, 1.5), a + "dkv.norm": vec(R, 1.0), a + "uk": lin(H * d, R, 1.5),
                      a + "uv": lin(H * dv, R), a + "o": lin(D, H * dv, 2.0)})
        if L["mlp"] is not None:
            ff = L["mlp"]["ff"]
            sublayer(p, 2)
            w.update({p + "mlp.gate": lin(ff, D, 1.5), p + "mlp.up": lin(ff, D, 1.5), p + "mlp.down": lin(D, ff)})
    return w


def run(cfg, w, tokens, collect_layers=False):
    """Logits of every position of one sequence (float64 [T, vocab]); with collect_layers also the sum of the streams after every layer."""
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
