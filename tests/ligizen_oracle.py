"""Plain, slow statement of a decoder of parallel layers (the Ligizen design), one function per mechanism, in float64 on the
CPU: whole sequences at once, no cache, no state carried between calls, nothing shared with the package."""
import math

import torch

DT = torch.float64
STEEP = 1.702                      # of the experts' gate


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def softcap(z, cap):
    return cap * torch.tanh(z / cap)


# --------------------------------------------------------------------------- rotation
def band_scaled(freq, s):
    """Frequencies with long wavelengths divided by the factor, those between the two bounds blended."""
    out = []
    for f in freq.tolist():
        wave = 2 * math.pi / f
        if wave < s["original"] / s["high"]:
            out.append(f)
        elif wave > s["original"] / s["low"]:
            out.append(f / s["factor"])
        else:
            t = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
            out.append((1 - t) * f / s["factor"] + t * f)
    return torch.tensor(out, dtype=DT)


def angles(T, rot):
    f = rot["base"] ** (-2 * torch.arange(rot["dims"] // 2, dtype=DT) / rot["dims"])
    if rot.get("scaling"):
        f = band_scaled(f, rot["scaling"])
    return torch.arange(T, dtype=DT)[:, None] * f


def rotate_half(x, a):
    """x [T, H, d]; dimension i of the first 2 n is paired with i + n."""
    n, c, s = a.shape[1], torch.cos(a)[:, None], torch.sin(a)[:, None]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], -1)


def rotate_pairs(x, a):
    """x [T, H, d]; dimensions 2i and 2i + 1 are a pair."""
    n, c, s = a.shape[1], torch.cos(a)[:, None], torch.sin(a)[:, None]
    u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
    out = x.clone()
    out[..., 0:2 * n:2], out[..., 1:2 * n:2] = u * c - v * s, v * c + u * s
    return out


# --------------------------------------------------------------------------- attention
def chunk_mask(T, size):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i // size == j // size)


def window_mask(T, size):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (i >= j) & (i - j < size)


def attend(q, k, v, scale, mask, sink=None):
    """q [T, H, d], k [T, G, d], v [T, G, n]; query head h reads key / value head h // (H / G); sink [H]: a score without
    key and value."""
    pick = torch.arange(q.shape[1]) // (q.shape[1] // k.shape[1])
    s = torch.einsum("qhd,khd->hqk", q, k[:, pick]) * scale
    s = s.masked_fill(~mask, -math.inf)
    if sink is not None:
        s = torch.cat([s, sink[:, None, None].expand(-1, q.shape[0], 1)], -1)
    p = torch.softmax(s, -1)[..., :k.shape[0]]
    return torch.einsum("hqk,khn->qhn", p, v[:, pick])


def keys_values(h, w, m, eps):
    T, G = h.shape[0], m["kv_heads"]
    k = (h @ w["k"].T + w["k.b"]).view(T, G, m["dim"])
    v = (h @ w["v"].T + w["v.b"]).view(T, G, m["vdim"])
    return rms(rotate_half(k, angles(T, m["rot"])), eps), v


def chunk_attention(h, w, m, eps, kv):
    T, H = h.shape[0], m["heads"]
    q = (h @ w["q"].T + w["q.b"]).view(T, H, m["dim"])
    q = rms(rotate_half(q, angles(T, m["rot"])), eps)
    o = attend(q, *kv, m["scale"], chunk_mask(T, m["mask"]["size"]))
    return (o * torch.sigmoid(h @ w["g"].T)[..., None]).reshape(T, -1) @ w["o"].T


def latent_attention(h, w, m, eps):
    T, H, R = h.shape[0], m["heads"], m["kv_rank"]
    a = angles(T, m["rot"])
    q = (rms(h @ w["dq"].T, eps) * w["dq.norm"] @ w["uq"].T).view(T, H, m["dim"] + m["rot_dim"])
    d = h @ w["dkv"].T
    c = rms(d[:, :R], eps) * w["dkv.norm"]
    k_rot = rotate_pairs(d[:, None, R:], a).expand(-1, H, -1)
    q = torch.cat([q[..., :m["dim"]], rotate_pairs(q[..., m["dim"]:], a)], -1)
    k = torch.cat([(c @ w["uk"].T).view(T, H, m["dim"]), k_rot], -1)
    v = (c @ w["uv"].T).view(T, H, m["vdim"])
    o = attend(q, k, v, m["scale"], window_mask(T, m["mask"]["size"]), w["sink"])
    return (o * torch.sigmoid(h @ w["g"].T)[..., None]).reshape(T, -1) @ w["o"].T


# --------------------------------------------------------------------------- feed-forward, token input
def silu_mlp(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def clamped_mlp(h, gate, up, down, limit):
    g, u = torch.clamp(h @ gate.T, max=limit), torch.clamp(h @ up.T, -limit, limit)
    return (g * torch.sigmoid(STEEP * g) * (u + 1)) @ down.T


def route(z, top):
    """Router logits of one token -> (experts, weights)."""
    s = torch.sigmoid(z)
    pick = sorted(range(len(z)), key=lambda e: -z[e].item())[:top]
    return pick, s[pick]


def experts(h, w, m):
    out, z = torch.zeros_like(h), h @ w["router"].T
    mats = lambda p: [w[p + n] for n in ("gate", "up", "down")]
    for t in range(h.shape[0]):
        for e, c in zip(*route(z[t], m["router"]["top"])):
            out[t] += clamped_mlp(c * h[t], *mats(f"e{e}."), m["expert"]["limit"])
    if m.get("shared"):
        out = out + torch.sigmoid(h @ w["shared.sg"].T) * clamped_mlp(h, *mats("shared."), m["shared"]["limit"])
    return out


def side_input(x, e, w, eps):
    y = (gelu_tanh(x @ w["side.gate"].T) * e) @ w["side.proj"].T
    return rms(y, eps) * w["side.norm"]


def under(w, p):
    return {k[len(p):]: v for k, v in w.items() if k.startswith(p)}


def forward(raw, weights, ids):
    """(logits [T, vocab], residual after every layer) of a whole sequence."""
    W = {k: v.to(DT) for k, v in weights.items()}
    eps, ids = raw["norm"]["eps"], torch.as_tensor(ids)
    x, taps, kvs = W["embed"][ids] * raw["embedding"]["scale"], [], {}
    for i, layer in enumerate(raw["layers"]):
        w, m, mlp = under(W, f"l{i}."), layer["mixer"], layer["mlp"]
        h, mix = layer_norm(x, w["norm1"], w["norm1.b"], eps), under(w, "mix.")
        if layer["type"] == "attention":
            j = m.get("kv_from")
            if j is None:
                j, kvs[i] = i, keys_values(h, mix, m, eps)
            y = chunk_attention(h, mix, m, eps, kvs[j])
        else:
            y = latent_attention(h, mix, m, eps)
        if mlp is not None:
            f = under(w, "mlp.")
            y = y + (silu_mlp(h, f["gate"], f["up"], f["down"]) if mlp["kind"] == "dense" else experts(h, f, mlp))
        x = x + y
        if raw.get("token_side"):
            n = raw["token_side"]["dim"]
            x = x + side_input(x, W["side.embed"][ids, i * n:(i + 1) * n], w, eps)
        taps.append(x)
    logits = layer_norm(x, W["final.norm"], W["final.norm.b"], eps) @ W["head"].T
    return softcap(logits, raw["logit_softcap"]), taps


# ----------------------------------------------------------------------------- small models for the tests
def small_config(width=96, vocab=160, layers="lcLk", mlps="dmsd", heads=4, kv_heads=2, dim=24, vdim=40, chunk=21, scale=None,
                 rot=16, scaling=(8.0, 1.0, 4.0, 64), lheads=3, ldim=20, lrot=8, lvdim=24, rank=40, q_rank=56, window=27,
                 lscale=None, ff=112, experts=6, top=2, eff=40, limit=1.2, sff=48, slimit=0.8, side=24, cap=20.0, escale=3.0,
                 eps=1e-5):
    """config.json contents.  Layers: 'l' latent attention, 'L' the same with other sizes, 'c' chunked attention, 'k' chunked
    attention on the keys of the last 'c' (with a chunk of its own); mlps: 'd' dense, 'm' routed with a shared expert, 's'
    routed without, '-' none."""
    specs, source = [], None
    for i, (c, f) in enumerate(zip(layers, mlps)):
        if c in "lL":
            kind, wide = "latent_attention", c == "L"
            m = {"heads": lheads + 2 * wide, "dim": ldim, "rot_dim": lrot, "vdim": lvdim + 8 * wide, "kv_rank": rank + 16 * wide,
                 "q_rank": q_rank, "mask": {"size": window + 10 * wide}, "scale": lscale or 2 * (ldim + lrot) ** -0.5,
                 "rot": {"base": 3000.0, "dims": lrot}}
        else:
            kind = "attention"
            m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk + 6 * (c == "k")},
                 "scale": scale or 2 * dim ** -0.5, "rot": {"base": 700.0, "dims": rot}}
            if scaling:
                m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
            if c == "k":
                m["kv_from"] = source
            else:
                source = i
        mlp = {"d": {"kind": "dense", "ff": ff}, "-": None}.get(f, {
            "kind": "moe", "expert": {"ff": eff, "limit": limit}, "router": {"experts": experts, "top": top}})
        if f == "m":
            mlp["shared"] = {"ff": sff, "limit": slimit}
        specs.append({"type": kind, "mixer": m, "mlp": mlp})
    return {"architecture": "Ligizen", "embedding": {"scale": escale}, "layers": specs, "logit_softcap": cap,
            "norm": {"eps": eps}, "token_side": {"dim": side}, "vocab": vocab, "width": width}


def small_weights(raw, shapes, seed=0):
    """bf16 tensors of the given name -> shape map, scaled so that every mechanism has a visible effect: scores of several
    units, sinks that take a share, clamps that bite, decided routers, biases of the size of what they are added to."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes.items():
        x, leaf = torch.randn(shape, generator=g), name.rsplit(".", 1)[-1]
        if name.endswith(".sink"):
            x = 1 + x
        elif leaf == "b":
            x = 0.5 * x
        elif leaf in ("norm1", "norm"):
            x = 1 + 0.3 * x
        elif leaf == "router":
            x = x * 4 / shape[-1] ** 0.5
        elif leaf in ("gate", "up") and ".side." not in name:
            x = x * 1.5 / shape[-1] ** 0.5
        elif len(shape) == 2 and name not in ("embed", "side.embed"):
            x = x / shape[-1] ** 0.5
        out[name] = x.to(torch.bfloat16)
    return out
