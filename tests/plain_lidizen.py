"""A plain, slow implementation of the Lidizen design in float64 on the CPU: whole sequences, no cache, one function
per mechanism, written from the design's equations and sharing no code with the package.

    x_t = LN_embed(E[token_t] + B[row_t])                  row_t from the pair (token_(t-1), token_t)
    z_1 = .. = z_n = x                                     ``streams`` copies
    per sub-layer f with a (in), b (out), M (mix, [from, to]):
        u = sum_s a_s z_s;  y = f(LN(u));  z_t <- sum_s M[s, t] z_s + b_t y        (all from the old streams)
    logits = E LN_final(sum_s z_s)

LN is a layer norm with a weight and no bias.  The mixer is a softmax attention over a sliding window and the
sequence's first tokens, whose heads' scores are mixed with one another before the softmax and whose values are mixed
with those of the first such layer; the feed-forward is a silu-gated unit with biases or a mixture of ungated experts.
"""
from __future__ import annotations

import torch

F64 = torch.float64


def layer_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    centred = x - x.mean(dim=-1, keepdim=True)
    return centred / torch.sqrt(centred.pow(2).mean(dim=-1, keepdim=True) + eps) * w


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps) * w


def silu(z: torch.Tensor) -> torch.Tensor:
    return z / (1.0 + torch.exp(-z))


def bigram_rows(tokens: list, buckets: int, mul_prev: int, mul_cur: int) -> list:
    """The row of the pair table of every token; the first token of a sequence has a row of its own, the last."""
    return [buckets if i == 0 else (tokens[i - 1] * mul_prev + tokens[i] * mul_cur) % buckets for i in range(len(tokens))]


def embed_tokens(W: dict, cfg: dict, tokens: list) -> torch.Tensor:
    x = W["embed"][torch.tensor(tokens)]
    bigram = (cfg.get("embedding") or {}).get("bigram")
    if bigram is not None:
        x = x + W["bigram"][torch.tensor(bigram_rows(tokens, bigram["buckets"], bigram["mul_prev"], bigram["mul_cur"]))]
    return layer_norm(x, W["embed.norm"], cfg["norm"]["eps"])


def read_streams(z: torch.Tensor, a: torch.Tensor) -> torch.Tensor:
    """z [T, n, W] -> [T, W]."""
    return sum(a[s] * z[:, s] for s in range(z.shape[1]))


def write_streams(z: torch.Tensor, y: torch.Tensor, mix: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    n = z.shape[1]
    return torch.stack([sum(mix[s, t] * z[:, s] for s in range(n)) + b[t] * y for t in range(n)], dim=1)


def rotate_pairs(x: torch.Tensor, positions: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """x [T, heads, D]: entries 2i and 2i + 1 of the first ``dims`` turn together by position * base^(-2i / dims)."""
    out = x.clone()
    for i in range(dims // 2):
        angle = positions * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(angle)[:, None], torch.sin(angle)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def visible(T: int, size, keep_first: int) -> torch.Tensor:
    """[T, T] bool: position i sees j <= i if it is nearer than ``size`` or one of the first ``keep_first``."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    near = torch.ones(T, T, dtype=torch.bool) if size is None else i - j < size
    return (j <= i) & (near | (j < keep_first))


def mix_scores(scores: torch.Tensor, talk: torch.Tensor) -> torch.Tensor:
    """scores [H, T, T]: head h gets sum_g talk[h, g] scores[g]."""
    return torch.stack([sum(talk[h, g] * scores[g] for g in range(scores.shape[0])) for h in range(scores.shape[0])])


def mix_values(v: torch.Tensor, first: torch.Tensor, lam: torch.Tensor) -> torch.Tensor:
    return (1.0 - lam) * v + lam * first


def attention(W: dict, p: str, m: dict, h: torch.Tensor, eps: float, first_values=None):
    """Returns (output, values as projected)."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ W[p + n].T + W[p + n + ".b"] for n in ("q", "k", "v"))
    projected = v
    q, k = rms_norm(q, W[p + "q.norm"], eps), rms_norm(k, W[p + "k.norm"], eps)
    q, k, v = q.view(T, H, D), k.view(T, G, D), v.view(T, G, V)
    rot = m.get("rot")
    if rot is not None:
        positions = torch.arange(T, dtype=F64)
        q, k = (rotate_pairs(x, positions, rot["base"], rot["dims"]) for x in (q, k))
    if first_values is not None:
        v = mix_values(v, first_values.view(T, G, V), W[p + "vmix"])
    per = H // G
    scores = torch.stack([q[:, head] @ k[:, head // per].T for head in range(H)]) * m["scale"]
    scores = mix_scores(scores, W[p + "talk"])
    mask = m.get("mask") or {}
    scores = scores.masked_fill(~visible(T, mask.get("size"), mask.get("keep_first", 0)), -float("inf"))
    weights = torch.softmax(scores, dim=-1)
    out = torch.stack([weights[head] @ v[:, head // per] for head in range(H)], dim=1)
    return out.reshape(T, H * V) @ W[p + "o"].T, projected


def dense_unit(W: dict, p: str, h: torch.Tensor) -> torch.Tensor:
    gate, up = h @ W[p + "gate"].T + W[p + "gate.b"], h @ W[p + "up"].T + W[p + "up.b"]
    return (silu(gate) * up) @ W[p + "down"].T + W[p + "down.b"]


def relu_squared_expert(W: dict, p: str, h: torch.Tensor) -> torch.Tensor:
    return torch.relu(h @ W[p + "up"].T).pow(2) @ W[p + "down"].T


def route(z: torch.Tensor, top: int):
    """z [T, E] logits: the ``top`` largest of every row and the softmax over those alone."""
    values, chosen = torch.topk(z, top, dim=-1)
    return chosen, torch.softmax(values, dim=-1)


def mixture(W: dict, p: str, mlp: dict, h: torch.Tensor) -> torch.Tensor:
    chosen, weight = route(h @ W[p + "router"].T + W[p + "router.b"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        w_e = (weight * (chosen == e)).sum(dim=-1)
        rows = w_e.nonzero()[:, 0]
        if len(rows):
            out[rows] += w_e[rows, None] * relu_squared_expert(W, f"{p}e{e}.", h[rows])
    return out


def forward(W: dict, cfg: dict, tokens: list, residuals: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of a whole sequence; ``residuals`` collects the sum of the streams after every layer."""
    W = {name: t.to(F64) for name, t in W.items()}
    eps = cfg["norm"]["eps"]
    n = cfg.get("streams", 1)
    z = embed_tokens(W, cfg, tokens)[:, None].expand(-1, n, -1).clone()
    first = None  # the values of the first layer that mixes them
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        h = layer_norm(read_streams(z, W[p + "hc1.in"]), W[p + "norm1"], eps)
        mixes = bool(m.get("v_mix"))
        y, values = attention(W, p + "mix.", m, h, eps, first if mixes else None)
        if mixes and first is None:
            first = values
        z = write_streams(z, y, W[p + "hc1.mix"], W[p + "hc1.out"])
        if mlp is not None:
            h = layer_norm(read_streams(z, W[p + "hc2.in"]), W[p + "norm2"], eps)
            y = dense_unit(W, p + "mlp.", h) if mlp["kind"] == "dense" else mixture(W, p + "mlp.", mlp, h)
            z = write_streams(z, y, W[p + "hc2.mix"], W[p + "hc2.out"])
        if residuals is not None:
            residuals.append(z.sum(dim=1))
    return layer_norm(z.sum(dim=1), W["final.norm"], eps) @ W["embed"].T
