"""The Tekarax design, plainly: float64, whole sequences, no cache, one function a mechanism.  It shares no code
with the engine; the GPU tests compare the engine with it.

``cfg`` is the configuration as ``config.json`` holds it, ``w`` a dict of float64 tensors by checkpoint name.
"""
from __future__ import annotations

import math

import torch

F = torch.float64


# --------------------------------------------------------------------------------------- norms, activations
def rms(x, eps):
    """x divided by its root mean square over the last dimension (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def layer_norm(x, weight, eps):
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


def relu_squared(z):
    return torch.clamp(z, min=0.0) ** 2


# ------------------------------------------------------------------------------------------------ rotation
def plain_frequencies(base, dims):
    return torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F)


def key_frequencies(rot):
    """f_i = base^(-2i/dims), i < dims/2; with ``scaling`` the long wavelengths are slowed down."""
    f = plain_frequencies(rot["base"], int(rot["dims"])).tolist()
    s = rot.get("scaling")
    if s:
        factor, low, high, original = float(s["factor"]), float(s["low"]), float(s["high"]), float(s["original"])
        for i, fi in enumerate(f):
            length = 2.0 * math.pi / fi
            if length < original / high:
                continue
            if length > original / low:
                f[i] = fi / factor
            else:
                blend = (original / length - low) / (high - low)
                f[i] = (1.0 - blend) * fi / factor + blend * fi
    return torch.tensor(f, dtype=F)


def rotate_halves(x, positions, freq):
    """x [T, heads, d]: entry i turns with entry i + n, i < n = len(freq), by positions * freq_i; entries from 2n on stay."""
    n = freq.numel()
    angle = positions.to(F)[:, None, None] * freq[None, None, :]
    c, s = torch.cos(angle), torch.sin(angle)
    u, v, rest = x[..., :n], x[..., n:2 * n], x[..., 2 * n:]
    return torch.cat([u * c - v * s, v * c + u * s, rest], dim=-1)


# ----------------------------------------------------------------------------------------------- attention
def softmax_attention(q, k, v, scale, window=None, sink=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; query i sees the keys j <= i, with ``window`` only those with
    i - j < window; query head h reads key/value head h // (H / G); ``sink`` [H]: exp(sink_h) joins head h's
    denominator."""
    T, H, _ = q.shape
    G = k.shape[1]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if window is not None:
        seen = seen & (i - j < window)
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~seen, -math.inf)
        if sink is not None:
            s = torch.cat([s, sink[h].expand(T, 1)], dim=1)
        p = torch.softmax(s, dim=-1)[:, :T]
        out[:, h] = p @ v[:, g]
    return out


def attention(m, w, p, h):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = (h @ w[p + "q"].T).view(T, H, D)
    k = (h @ w[p + "k"].T).view(T, G, D)
    v = (h @ w[p + "v"].T).view(T, G, V)
    freq = key_frequencies(m["rot"])
    q, k = rotate_halves(q, pos, freq), rotate_halves(k, pos, freq)
    turn = plain_frequencies(m["rot"]["base"], V)  # the values turn too, over all their entries, never slowed down
    v = rotate_halves(v, pos, turn)
    o = softmax_attention(q, k, v, float(m["scale"]), sink=w[p + "sink"])
    o = rotate_halves(o, -pos, turn)  # ... and each output turns back by its own position
    o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]  # one number a head
    return o.reshape(T, H * V) @ w[p + "o"].T


def latent_attention(m, w, p, h, eps):
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, D)
    c = rms(h @ w[p + "dkv"].T, eps) * w[p + "dkv.norm"]
    k = (c @ w[p + "uk"].T).view(T, H, D)
    v = (c @ w[p + "uv"].T).view(T, H, V)
    o = softmax_attention(q, k, v, float(m["scale"]), window=int(m["mask"]["size"]))
    return o.reshape(T, H * V) @ w[p + "o"].T


# --------------------------------------------------------------------------------------------- recurrence
def token_shift(h, mu):
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def wkv_scan(r, k, v, decay, u):
    """r, k, v, decay [T, H, D], u [H, D]: o_t = (S + diag(u) k v^T)^T r, then S <- diag(decay) S + k v^T."""
    T, H, D = r.shape
    o = torch.zeros(T, H, v.shape[2], dtype=F)
    for n in range(H):
        S = torch.zeros(D, v.shape[2], dtype=F)
        for t in range(T):
            kv = torch.outer(k[t, n], v[t, n])
            o[t, n] = (S + u[n][:, None] * kv).T @ r[t, n]
            S = decay[t, n][:, None] * S + kv
    return o


def wkv(m, w, p, h, eps):
    T = h.shape[0]
    H, D = m["heads"], m["dim"]
    mix = {c: token_shift(h, w[p + "mu." + c]) for c in "rkvgw"}
    r, k, v = ((mix[c] @ w[p + c].T).view(T, H, D) for c in "rkv")
    gate = silu(mix["g"] @ w[p + "g"].T)
    z = torch.tanh(mix["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]
    decay = torch.exp(-torch.exp(z)).view(T, H, D)
    o = rms(wkv_scan(r, k, v, decay, w[p + "u"]), eps).reshape(T, H * D)
    return (o * w[p + "norm"] * gate) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------- feed-forward
def dense_unit(w, p, h):
    return relu_squared(h @ w[p + "up"].T + w[p + "up.b"]) @ w[p + "down"].T + w[p + "down.b"]


def expert(w, p, h):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(mlp, w, p, h):
    """(chosen experts [T, top], weights [T, top]) best first."""
    s = torch.sigmoid(h @ w[p + "router"].T)
    weight, chosen = torch.sort(s, dim=-1, descending=True, stable=True)
    top = int(mlp["router"]["top"])
    return chosen[:, :top], weight[:, :top]


def mixture(mlp, w, p, h):
    chosen, weight = route(mlp, w, p, h)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(chosen.shape[1]):
            out[t] += expert(w, f"{p}e{int(chosen[t, j])}.", weight[t, j] * h[t:t + 1])[0]
    if mlp.get("shared"):
        out = out + expert(w, p + "shared.", h)
    return out


def feed_forward(mlp, w, p, h):
    return dense_unit(w, p, h) if mlp["kind"] == "dense" else mixture(mlp, w, p, h)


# -------------------------------------------------------------------------------------------------- model
def layer_runs(cfg):
    """The layers in the order they run: (layer, number of the pass that starts right before it, or None)."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    runs = [(i, None) for i in range(start)]
    for t in range(times):
        runs += [(i, t if i == start else None) for i in range(start, stop)]
    return runs + [(i, None) for i in range(stop, n)]


def sublayer(w, x, eps, norm_in, norm_out, gate, f):
    h = layer_norm(x, w[norm_in], eps)
    y = f(h) * torch.sigmoid(h @ w[gate].T + w[gate + ".b"])
    return x + layer_norm(y, w[norm_out], eps)


def layer(cfg, w, i, x):
    spec, eps = cfg["layers"][i], float(cfg["norm"]["eps"])
    p, m = f"l{i}.", spec["mixer"]
    mixers = {"attention": lambda h: attention(m, w, p + "mix.", h),
              "wkv": lambda h: wkv(m, w, p + "mix.", h, eps),
              "latent_attention": lambda h: latent_attention(m, w, p + "mix.", h, eps)}
    x = sublayer(w, x, eps, p + "norm1", p + "norm1b", p + "rg1", mixers[spec["type"]])
    if spec.get("mlp") is not None:
        x = sublayer(w, x, eps, p + "norm2", p + "norm2b", p + "rg2", lambda h: feed_forward(spec["mlp"], w, p + "mlp.", h))
    return x


def forward(cfg, w, ids, streams=False):
    """Logits [T, vocab] of one sequence; ``streams``: also the stream after every layer run."""
    eps = float(cfg["norm"]["eps"])
    x, seen = w["embed"][torch.as_tensor(ids)], []
    for i, began in layer_runs(cfg):
        if began is not None:
            x = x + w["loop.step"][began]
        x = layer(cfg, w, i, x)
        seen.append(x)
    logits = layer_norm(x, w["final.norm"], eps) @ w["head"].T
    return (logits, torch.stack(seen)) if streams else logits
