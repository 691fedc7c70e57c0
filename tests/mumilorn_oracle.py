"""Plain, slow statement of a decoder of pre-norm layers (the Mumilorn design), one function per mechanism, in float64 on
the CPU: whole sequences at once, no cache, no state carried between calls, nothing shared with the package."""
import math

import torch

DT = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def pre_norm(x, w, eps):
    """The weight is stored as its difference from one."""
    return rms(x, eps) * (1 + w)


def silu(z):
    return z * torch.sigmoid(z)


# --------------------------------------------------------------------------- recurrences
def linear_attention(q, k, v, a):
    """q, k, a [T, H, d], v [T, H, n] -> [T, H, n]: row c of the state is multiplied by a_t[c], then k_t v_t^T is added, then
    it is read with q_t."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def bonus_attention(r, k, v, w, u):
    """r, k, w [T, H, d], v [T, H, n], u [H, d]: read before the decay, the current token through the bonus u."""
    T, H, d = r.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=r.dtype)
    out = []
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out.append(((S + u[:, :, None] * kv) * r[t][:, :, None]).sum(1))
        S = w[t][:, :, None] * S + kv
    return torch.stack(out)


def sigmoid_root_decay(z, tau):
    return torch.sigmoid(z) ** (1 / tau)


def double_exp_decay(z):
    return torch.exp(-torch.exp(z))


def gla(h, w, m, eps):
    T, H, d, n = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T * d ** -0.5).view(T, H, d)
    k = (h @ w["k"].T).view(T, H, d)
    v = (h @ w["v"].T).view(T, H, n)
    a = sigmoid_root_decay(h @ w["a1"].T @ w["a2"].T + w["a2.b"], m["tau"]).view(T, H, d)
    o = rms(linear_attention(q, k, v, a), eps) * w["norm"]
    return (o.reshape(T, -1) * silu(h @ w["g"].T)) @ w["o"].T


def shifted(h):
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


def token_mix(h, mu):
    return h + (shifted(h) - h) * mu


def rwkv(h, w, m, eps):
    T, H, d = h.shape[0], m["heads"], m["dim"]
    x = {n: token_mix(h, w["mu." + n]) for n in "rkvgw"}
    r, k, v = ((x[n] @ w[n].T).view(T, H, d) for n in "rkv")
    decay = double_exp_decay(torch.tanh(x["w"] @ w["w1"].T) @ w["w2"].T + w["w0"]).view(T, H, d)
    o = rms(bonus_attention(r, k, v, decay, w["u"]), eps).reshape(T, -1)
    return (o * w["norm"] * silu(x["g"] @ w["g"].T)) @ w["o"].T


# --------------------------------------------------------------------------- attention
def window_mask(T, size):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (i >= j) & (i - j < size)


def softmax_attention(q, k, v, scale, mask):
    """q [T, H, d], k [T, G, d], v [T, G, n]; query head h reads key / value head h // (H / G)."""
    pick = torch.arange(q.shape[1]) // (q.shape[1] // k.shape[1])
    s = torch.einsum("qhd,khd->hqk", q, k[:, pick]) * scale
    return torch.einsum("hqk,khn->qhn", torch.softmax(s.masked_fill(~mask, -math.inf), -1), v[:, pick])


def row_norm(x, w, eps):
    """All heads of a token normed together."""
    return rms(x, eps) * w


def window_attention(h, w, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = row_norm(h @ w["q"].T, w["q.norm"], eps).view(T, H, m["dim"])
    k = row_norm(h @ w["k"].T, w["k.norm"], eps).view(T, G, m["dim"])
    v = (h @ w["v"].T).view(T, G, m["vdim"])
    o = softmax_attention(q, k, v, m["scale"], window_mask(T, m["mask"]["size"])).reshape(T, -1)
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def under(w, p):
    return {k[len(p):]: v for k, v in w.items() if k.startswith(p)}


def parallel(h, w, m, eps):
    return (m["left_scale"] * window_attention(h, under(w, "left."), m["left"], eps)
            + m["right_scale"] * rwkv(h, under(w, "right."), m["right"], eps))


# --------------------------------------------------------------------------- feed-forward
def squared_relu_mlp(h, up, down):
    return torch.relu(h @ up.T) ** 2 @ down.T


def silu_mlp(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def route(z, top, groups, scale):
    """Router logits of one token -> (experts, weights)."""
    s = torch.softmax(z, 0)
    allowed = range(len(z))
    if groups:
        n = len(z) // groups["count"]
        best = sorted(range(groups["count"]), key=lambda g: -max(s[g * n:(g + 1) * n].tolist()))[:groups["keep"]]
        allowed = [e for e in allowed if e // n in best]
    pick = sorted(allowed, key=lambda e: -s[e].item())[:top]
    w = s[pick] / (s[pick].sum() + 1e-20) * scale
    return pick, w


def experts(h, w, m):
    r, out = m["router"], torch.zeros_like(h)
    z = h @ w["router"].T
    for t in range(h.shape[0]):
        for e, c in zip(*route(z[t], r["top"], r.get("groups"), r["scale"])):
            out[t] += c * silu_mlp(h[t], *(w[f"e{e}.{n}"] for n in ("gate", "up", "down")))
    return out


def forward(raw, weights, ids):
    """(logits [T, vocab], residual after every layer) of a whole sequence."""
    W = {k: v.to(DT) for k, v in weights.items()}
    eps = raw["norm"]["eps"]
    x, taps = W["embed"][torch.as_tensor(ids)], []
    for i, layer in enumerate(raw["layers"]):
        w = under(W, f"l{i}.")
        mixer = {"gla": gla, "parallel": parallel}[layer["type"]]
        x = x + mixer(pre_norm(x, w["norm1"], eps), under(w, "mix."), layer["mixer"], eps)
        if layer["mlp"]:
            h, m = pre_norm(x, w["norm2"], eps), layer["mlp"]
            if m["kind"] == "dense":
                x = x + squared_relu_mlp(h, w["mlp.up"], w["mlp.down"])
            else:
                x = x + experts(h, under(w, "mlp."), m)
        taps.append(x)
    return pre_norm(x, W["final.norm"], eps) @ W["embed"].T, taps


# ----------------------------------------------------------------------------- small models for the tests
def small_config(width=96, vocab=160, layers="gpg", mlps="dmd", heads=4, kv_heads=2, dim=24, vdim=40, window=21, scale=None,
                 lheads=3, ldim=20, lvdim=28, tau=8.0, rheads=2, rdim=24, left_scale=0.6, right_scale=1.3, ff=112, experts=6,
                 top=2, eff=40, groups=(3, 2), rscale=1.7, eps=1e-5):
    """config.json contents: layers 'g' gated linear attention, 'p' parallel; mlps 'd' dense, 'm' routed, '-' none."""
    specs = []
    for c, f in zip(layers, mlps):
        if c == "g":
            kind, m = "gla", {"heads": lheads, "dim": ldim, "vdim": lvdim, "tau": tau}
        else:
            kind = "parallel"
            m = {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
                          "scale": scale or dim ** -0.5},
                 "right": {"heads": rheads, "dim": rdim}, "left_scale": left_scale, "right_scale": right_scale}
        mlp = {"d": {"kind": "dense", "ff": ff}, "-": None,
               "m": {"kind": "moe", "expert": {"ff": eff},
                     "router": {"experts": experts, "top": top, "scale": rscale,
                                "groups": {"count": groups[0], "keep": groups[1]} if groups else None}}}[f]
        specs.append({"type": kind, "mixer": m, "mlp": mlp})
    return {"architecture": "Mumilorn", "layers": specs, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def small_weights(raw, shapes, seed=0):
    """bf16 tensors of the given name -> shape map, scaled so that every mechanism has a visible effect: slow decays with a
    few fast channels, scores of several units, mixes over the whole range, strong bonus, decided routers."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes.items():
        x, leaf = torch.randn(shape, generator=g), name.rsplit(".", 1)[-1]
        if leaf in ("norm1", "norm2") or name == "final.norm":
            x = 0.3 * x
        elif name.endswith(("q.norm", "k.norm")):
            x = 1.6 + 0.4 * x
        elif leaf == "norm":
            x = 1 + 0.3 * x
        elif ".mu." in name:
            x = torch.rand(shape, generator=g)
        elif leaf == "w0":
            x = -2.5 + 1.5 * x
        elif leaf == "b":
            x = 1 + 1.5 * x
        elif leaf == "u":
            x = 1.5 * x
        elif leaf == "router":
            x = x * 4 / shape[-1] ** 0.5
        elif leaf in ("w2", "a2"):
            x = x / shape[-1] ** 0.5
        elif len(shape) == 2 and name != "embed":
            x = x / shape[-1] ** 0.5
        out[name] = x.to(torch.bfloat16)
    return out
