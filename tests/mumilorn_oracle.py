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
