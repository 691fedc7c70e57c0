"""Plain, slow statement of a decoder of layers normed before and after each sublayer (the Redodra design), one function per
mechanism, in float64 on the CPU: whole sequences at once, no cache, no state carried between calls, nothing shared with the
package."""
import math

import torch

DT = torch.float64


# --------------------------------------------------------------------------- norms, activations
def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def tanh_norm(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.logaddexp(z, torch.zeros_like(z))


def softcap(z, cap):
    return cap * torch.tanh(z / cap)


def xielu(z, p, q):
    pos = softplus(p) * z * z + z / 2
    neg = (0.5 + softplus(q)) * (torch.expm1(z) - z) + z / 2
    return torch.where(z > 0, pos, neg)


def mlp(h, up, down, act):
    return xielu(h @ up.T, act[0], act[1]) @ down.T


def depth_average(coef, xs):
    return sum(c * x for c, x in zip(coef, xs))


# --------------------------------------------------------------------------- attention
def rotate_pairs(x, base, dims):
    """x [T, H, d]: pairs (2i, 2i + 1) of the first `dims` dimensions turned by position * base^(-2i / dims)."""
    T, out = x.shape[0], x.clone()
    for i in range(dims // 2):
        a = torch.arange(T, dtype=x.dtype)[:, None] * base ** (-2 * i / dims)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


def distances(T):
    return torch.arange(T)[:, None] - torch.arange(T)[None, :]


def causal_mask(T):
    return distances(T) >= 0


def window_mask(T, size, keep_first):
    """The last `size` tokens and the first `keep_first` ones."""
    d = distances(T)
    return (d >= 0) & ((d < size) | (torch.arange(T)[None, :] < keep_first))


def distance_bias(T, r1, r2):
    """[H, T, T]: what a score loses with the distance."""
    d = distances(T).clamp(min=0).to(DT)
    return r1[:, None, None] * torch.log1p(r2[:, None, None] * d)


def softmax_attention(q, k, v, scale, mask, cap=0.0, bias=None, sink=None):
    """q [T, H, d], k [T, G, d], v [T, G, n] -> [T, H, n]; query head h reads key / value head h // (H / G); sink [H]: the
    logarithm of one more addend of the denominator."""
    pick = torch.arange(q.shape[1]) // (q.shape[1] // k.shape[1])
    s = torch.einsum("qhd,khd->hqk", q, k[:, pick]) * scale
    if cap:
        s = softcap(s, cap)
    if bias is not None:
        s = s - bias
    s = s.masked_fill(~mask, -math.inf)
    if sink is not None:
        s = torch.cat([s, sink[:, None, None].expand(*s.shape[:2], 1)], -1)
    return torch.einsum("hqk,khn->qhn", torch.softmax(s, -1)[..., :len(k)], v[:, pick])


def keys_values(h, w, m):
    k = rotate_pairs((h @ w["k"].T).view(len(h), m["kv_heads"], m["dim"]), m["rot"]["base"], m["rot"]["dims"])
    return k, (h @ w["v"].T).view(len(h), m["kv_heads"], m["vdim"])


def attention(h, w, m, kv):
    T = len(h)
    q = rotate_pairs((h @ w["q"].T).view(T, m["heads"], m["dim"]), m["rot"]["base"], m["rot"]["dims"])
    o = softmax_attention(q, *kv, m["scale"], causal_mask(T), m.get("softcap"), sink=w["sink"])
    return (o * torch.sigmoid(h @ w["g"].T)[..., None]).reshape(T, -1) @ w["o"].T


def window_attention(h, w, m):
    T, H, G = len(h), m["heads"], m["kv_heads"]
    q = (h @ w["q"].T + w["q.b"]).view(T, H, m["dim"])
    k = (h @ w["k"].T + w["k.b"]).view(T, G, m["dim"])
    v = (h @ w["v"].T + w["v.b"]).view(T, G, m["vdim"])
    mask = window_mask(T, m["mask"]["size"], m["mask"]["keep_first"])
    o = softmax_attention(q, k, v, m["scale"], mask, m.get("softcap"), distance_bias(T, w["r1"], w["r2"]))
    return o.reshape(T, -1) @ w["o"].T + w["o.b"]


# --------------------------------------------------------------------------- recurrences
def short_conv(x, w, b=None):
    """x [T, C], w [C, taps], the last column for the current token."""
    taps = w.shape[1]
    past = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    y = sum(past[i:i + len(x)] * w[:, i] for i in range(taps))
    return y if b is None else y + b


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, g, beta):
    """q, k [T, H, d], v [T, H, n], g and beta [T, H] -> [T, H, n]."""
    S, out = torch.zeros(*q.shape[1:], v.shape[-1], dtype=q.dtype), []
    for t in range(len(q)):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdn,hd->hn", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdn,hd->hn", S, q[t]))
    return torch.stack(out)


def delta(h, w, m, eps):
    T, H, G, d, n = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_conv(h @ w[c].T, w[c + ".conv"])) for c in "qkv")
    pick = torch.arange(H) // (H // G)
    q = unit(q.view(T, G, d))[:, pick] * d ** -0.5
    k = unit(k.view(T, G, d))[:, pick]
    beta = torch.sigmoid(h @ w["b"].T)
    g = torch.exp(-torch.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    o = rms(delta_rule(q, k, v.view(T, H, n), g, beta), eps) * w["norm"]
    return (o.reshape(T, -1) * silu(h @ w["g"].T)) @ w["o"].T


def state_space(x, B, C, dt, A):
    """x [T, H, n], B and C [T, H, N], dt [T, H], A [H] (negative) -> [T, H, n]."""
    S, out = torch.zeros(x.shape[1], B.shape[2], x.shape[2], dtype=x.dtype), []
    for t in range(len(x)):
        S = torch.exp(A * dt[t])[:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        out.append(torch.einsum("hdn,hd->hn", S, C[t]))
    return torch.stack(out)


def mamba2(h, w, m, eps):
    T, H, n, N, G = len(h), m["heads"], m["vdim"], m["state"], m["groups"]
    z, xbc, dt = (h @ w["in"].T).split([H * n, H * n + 2 * G * N, H], -1)
    x, B, C = silu(short_conv(xbc, w["conv"], w["conv.b"])).split([H * n, G * N, G * N], -1)
    pick, x = torch.arange(H) // (H // G), x.reshape(T, H, n)
    dt = softplus(dt + w["dt_bias"])
    y = state_space(x, B.reshape(T, G, N)[:, pick], C.reshape(T, G, N)[:, pick], dt, -torch.exp(w["A_log"]))
    y = (y + w["D"][:, None] * x).reshape(T, -1) * silu(z)
    y = rms(y.view(T, m["norm_groups"], -1), eps).reshape(T, -1) * w["norm"]
    return y @ w["o"].T


def under(w, p):
    return {k[len(p):]: v for k, v in w.items() if k.startswith(p)}


def parallel(h, w, m, eps):
    left = window_attention(h, under(w, "left."), m["left"])
    right = mamba2(h, under(w, "right."), m["right"], eps)
    return (rms(left, eps) * w["left.out"] + rms(right, eps) * w["right.out"]) / 2


# --------------------------------------------------------------------------- the model
def forward(raw, weights, ids):
    """(logits [T, vocab], what goes on after every layer) of a whole sequence."""
    W = {k: v.to(DT) for k, v in weights.items()}
    norm = lambda x, name: tanh_norm(x, W[name + ".alpha"], W[name], W[name + ".b"])
    eps = raw["norm"]["eps"]
    x = W["embed"][torch.as_tensor(ids)]
    results, taps, kvs = [x], [], {}
    for i, layer in enumerate(raw["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h, mix = norm(x, p + "norm1"), under(W, p + "mix.")
        if layer["type"] == "attention":
            j = m.get("kv_from")
            if j is None:
                j, kvs[i] = i, keys_values(h, mix, m)
            y = attention(h, mix, m, kvs[j])
        else:
            y = {"delta": delta, "parallel": parallel}[layer["type"]](h, mix, m, eps)
        x = x + norm(y, p + "norm1b")
        if layer["mlp"] is not None:
            y = mlp(norm(x, p + "norm2"), W[p + "mlp.up"], W[p + "mlp.down"], W[p + "mlp.act"])
            x = x + norm(y, p + "norm2b")
        results.append(x)
        x = depth_average(W[p + "dwa"], results)
        taps.append(x)
    return norm(x, "final.norm") @ W["head"].T, taps


# ----------------------------------------------------------------------------- small models for the tests
def small_config(width=88, vocab=150, layers="dpakp", mlps="dd-dd", ff=104, heads=4, kv_heads=2, dim=24, vdim=40, rot=16, base=900.0,
                 cap=9.0, scale=None, dheads=4, dkv=2, ddim=16, dvdim=24, dconv=3, lheads=6, lkv=2, ldim=20, lvdim=28, window=19,
                 first=5, lcap=7.0, lscale=None, rheads=6, groups=3, state=12, rvdim=20, rconv=4, parts=2, eps=1e-4):
    """config.json contents.  Layers: 'd' delta rule, 'D' the same with other sizes, 'p' attention beside the state-space mixer, 'a'
    attention, 'k' attention on the keys of the last 'a'; mlps: 'd' dense, '-' none."""
    specs, source = [], None
    for i, (c, f) in enumerate(zip(layers, mlps)):
        if c in "dD":
            kind, n = "delta", c == "D"
            m = {"heads": dheads * (1 + n), "kv_heads": dkv, "dim": ddim + 8 * n, "vdim": dvdim, "conv": dconv + n}
        elif c == "p":
            kind = "parallel"
            m = {"left": {"heads": lheads, "kv_heads": lkv, "dim": ldim, "vdim": lvdim, "scale": lscale or 1.5 * ldim ** -0.5,
                          "softcap": lcap, "mask": {"size": window, "keep_first": first}},
                 "right": {"heads": rheads, "groups": groups, "state": state, "vdim": rvdim, "conv": rconv, "norm_groups": parts}}
        else:
            kind = "attention"
            m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 1.5 * dim ** -0.5, "softcap": cap,
                 "rot": {"base": base, "dims": rot}}
            if c == "k":
                m["kv_from"] = source
            else:
                source = i
        specs.append({"type": kind, "mixer": m, "mlp": {"kind": "dense", "ff": ff} if f == "d" else None})
    return {"architecture": "Redodra", "layers": specs, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def small_weights(raw, shapes, seed=0):
    """bf16 tensors of the given name -> shape map, scaled so that every mechanism has a visible effect: scores of several
    units, sinks that take a share, decays from fast to slow, averages that mix all depths."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes.items():
        x, leaf = torch.randn(shape, generator=g), name.rsplit(".", 1)[-1]
        if name.endswith(".mix.sink"):
            x = 1 + x
        elif leaf in ("r1", "r2"):
            x = torch.rand(shape, generator=g) * (0.8 if leaf == "r1" else 0.3) + 0.1
        elif leaf == "alpha":
            x = 0.5 + 0.5 * torch.rand(shape, generator=g)
        elif leaf in ("A_log", "dt_bias"):
            x = x - 1
        elif leaf == "dwa":
            x = 0.3 * x
            x[-1] += 1
        elif leaf == "conv":
            x = x / shape[-1] ** 0.5
        elif len(shape) == 1 and leaf != "act":
            x = 0.4 * x + (leaf in ("norm1", "norm2", "norm1b", "norm2b", "norm", "out", "D"))
        elif len(shape) == 2 and name != "embed":
            x = x * (2.0 if leaf in ("q", "k") else 1.2) / shape[-1] ** 0.5
        out[name] = x.to(torch.bfloat16)
    return out
