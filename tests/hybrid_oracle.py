"""Plain, slow statement of the layers in `nkipy_b200/models/hybrid.py`, one function per mechanism, in float64 on the
CPU: whole sequences at once, no cache, no state carried between calls, nothing shared with the package."""
import math

import torch

DT = torch.float64


def embed(table, ids, scale):
    return table[torch.as_tensor(ids)] * scale


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def group_norm(x, w, groups, eps):
    parts = x.reshape(*x.shape[:-1], groups, -1)
    return rms(parts, eps).reshape(x.shape) * w


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def gated_mlp(h, gate, up, down):
    return (gelu_tanh(h @ gate.T) * (h @ up.T)) @ down.T


def result_gate(h, w, b):
    return torch.sigmoid(h @ w.T + b)


def forget_gate(z, bias, lower):
    return lower + (1 - lower) * torch.sigmoid(z + bias)


def recurrence(q, f, v):
    """q, f [T, heads, dim], v [T, heads, vdim] -> o [T, heads, vdim], with S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = f[t][:, :, None] * S + (1 - f[t])[:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def hgrn2(h, w, m, eps):
    T = h.shape[0]
    u = h @ w["q"].T
    q = (u * torch.sigmoid(u)).view(T, m["heads"], m["dim"])
    f = forget_gate(h @ w["f"].T, w["f.b"], w["lower"]).view(T, m["heads"], m["dim"])
    v = (h @ w["v"].T).view(T, m["heads"], m["vdim"])
    o = rms(recurrence(q, f, v), eps) * w["norm"]
    return o.reshape(T, -1) @ w["o"].T


def yarn(rot):
    """(frequencies, multiplier of cos and sin) of a rotation with optional scaling."""
    n, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2 * i / n) for i in range(n // 2)]
    if not sc:
        return torch.tensor(f, dtype=DT), 1.0

    def dim(t):
        return n * math.log(sc["original"] / (2 * math.pi * t)) / (2 * math.log(base))

    lo, hi = max(math.floor(dim(sc["fast"])), 0), min(math.ceil(dim(sc["slow"])), n - 1)
    ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(n // 2)]
    f = [x / sc["factor"] * r + x * (1 - r) for x, r in zip(f, ramp)]
    return torch.tensor(f, dtype=DT), 0.1 * math.log(sc["factor"]) + 1


def rotate(x, rot, positions):
    """x [T, ..., dim]: pairs (2i, 2i + 1) of the first rot dims turned by position times frequency."""
    f, mult = yarn(rot)
    a = torch.as_tensor(positions, dtype=DT)[:, None] * f
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (f.numel(),)
    c, s = (a.cos() * mult).view(shape), (a.sin() * mult).view(shape)
    out = x.clone()
    u, v = x[..., 0:rot["dims"]:2], x[..., 1:rot["dims"]:2]
    out[..., 0:rot["dims"]:2] = u * c - v * s
    out[..., 1:rot["dims"]:2] = v * c + u * s
    return out


def capped(s, cap):
    return cap * torch.tanh(s / cap) if cap else s


def score_map(q, k, v, scale, cap):
    """One causal map: q, k [T, H, dim], v [T, H, vdim] (heads already repeated)."""
    T = q.shape[0]
    s = capped(torch.einsum("qhd,khd->hqk", q, k) * scale, cap)
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), -math.inf)
    return torch.einsum("hqk,khv->qhv", torch.softmax(s, -1), v)


def map_weight(w, diff):
    return torch.exp((w["lq1"] * w["lk1"]).sum()) - torch.exp((w["lq2"] * w["lk2"]).sum()) + diff


def combine(a1, a2, lam, diff, eps):
    return rms(a1 - lam * a2, eps) * (1 - diff)


def diff_attention(h, w, m, eps):
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = rotate((h @ w["q"].T).view(T, H, 2, d), m["rot"], range(T))
    k = rotate((h @ w["k"].T).view(T, G, 2, d), m["rot"], range(T))
    v = (h @ w["v"].T).view(T, G, m["vdim"])
    pick = torch.arange(H) // (H // G)
    a = [score_map(q[:, :, i], k[:, pick, i], v[:, pick], m["scale"], m.get("softcap")) for i in (0, 1)]
    o = combine(a[0], a[1], map_weight(w, m["diff"]), m["diff"], eps)
    return o.reshape(T, -1) @ w["o"].T


def forward(raw, weights, ids):
    """(logits [T, vocab], residual after every layer run) of a whole sequence."""
    W = {k: v.to(DT) for k, v in weights.items()}
    eps, groups = raw["norm"]["eps"], raw["norm"]["groups"]
    e = embed(W["embed"], ids, raw["embedding"]["scale"])
    x, taps, n = e, [], len(raw["layers"])
    lp = raw.get("loop") or {"start": n, "stop": n, "times": 1}
    order = [(i, None) for i in range(lp["start"])]
    for t in range(lp["times"]):
        order += [(i, t) for i in range(lp["start"], lp["stop"])]
    order += [(i, None) for i in range(lp["stop"], n)]
    for i, t in order:
        if t is not None and i == lp["start"]:
            if t > 0:
                x = x + e
            x = x + W["loop.step"][t]
        layer, p = raw["layers"][i], f"l{i}."
        mix = {k[len(p) + 4:]: v for k, v in W.items() if k.startswith(p + "mix.")}
        h1 = group_norm(x, W[p + "norm1"], groups, eps)
        mixer = hgrn2 if layer["type"] == "hgrn2" else diff_attention
        y = mixer(h1, mix, layer["mixer"], eps) * result_gate(h1, W[p + "rg1"], W[p + "rg1.b"])
        if layer["mlp"]:
            h2 = group_norm(x, W[p + "norm2"], groups, eps)
            y = y + (gated_mlp(h2, W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"])
                     * result_gate(h2, W[p + "rg2"], W[p + "rg2.b"]))
        x = x + y
        taps.append(x)
    return group_norm(x, W["final.norm"], groups, eps) @ W["head"].T, taps


# ----------------------------------------------------------------------------- small models for the tests
def small_config(width=96, vocab=160, groups=3, layers="rar", loop=None, heads=4, kv_heads=2, dim=24, vdim=40, rdims=16,
                 rheads=3, rdim=20, rvdim=28, ff=112, softcap=8.0, scaling=True, no_ff=(), diff=0.4, scale=None,
                 eps=1e-5, emb=2.0):
    """config.json contents: 'r' recurrence, 'a' attention; layers whose index is in no_ff have no feed-forward."""
    specs = []
    for i, c in enumerate(layers):
        if c == "r":
            m = {"heads": rheads, "dim": rdim, "vdim": rvdim}
        else:
            rot = {"base": 10000.0, "dims": rdims}
            if scaling:
                rot["scaling"] = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}
            m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "diff": diff,
                 "scale": scale or dim ** -0.5, "softcap": softcap, "rot": rot}
        specs.append({"type": "hgrn2" if c == "r" else "attention", "mixer": m,
                      "mlp": None if i in no_ff else {"kind": "dense", "ff": ff}})
    raw = {"architecture": "Tolenex", "embedding": {"scale": emb}, "layers": specs,
           "norm": {"eps": eps, "groups": groups}, "vocab": vocab, "width": width}
    if loop:
        raw["loop"] = dict(zip(("start", "stop", "times"), loop))
    return raw


def small_weights(raw, shapes, seed=0):
    """bf16 tensors of the given name -> shape map, scaled so that every mechanism has a visible effect: forget gates
    near one (long memory), score differences of several units, gates and map weights away from their centres."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes.items():
        x = torch.randn(shape, generator=g)
        if name.endswith(("norm1", "norm2", ".norm")):
            x = 1 + 0.2 * x
        elif name.endswith("lower"):
            x = 0.5 + 0.45 * torch.rand(shape, generator=g)
        elif name.endswith("f.b"):
            x = 1.5 + x
        elif name.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            x = 0.25 * x
        elif name.endswith((".b", "loop.step")):
            x = 0.7 * x
        elif name.endswith(("mix.q", "mix.k")):
            x = x * 1.6 / shape[-1] ** 0.5
        elif len(shape) == 2:
            x = x / shape[-1] ** 0.5
        out[name] = x.to(torch.bfloat16)
    return out
