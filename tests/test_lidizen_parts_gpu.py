"""Each mechanism of the Lidizen design alone: the kernels and parts against the plain functions of tests/plain_lidizen.py, at
sizes of their own, with inputs designed so that a fault shows (keys just inside and just outside the window and the kept
first tokens, page 0 and every page that may be given back full of NaN, mixing matrices far from the identity, the last
token of an earlier step, an expert whose choice hangs on the router's bias)."""
import pytest
import torch

import plain_lidizen as plain
from test_kilatar_parts_gpu import DEV, TORCH, Ctx, _paged, close, rand

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
i32 = lambda values: torch.as_tensor(values, dtype=torch.int32).to(DEV)


def spread(q, talk, G):
    """q [T, H, P], talk [H, H] -> [T, H, G, P]: head h's piece for KV head c is sum over the heads g of c of talk[h, g] q_g."""
    T, H, P = q.shape
    return torch.einsum("hcj,tcjp->thcp", talk.view(H, G, H // G), q.view(T, G, H // G, P))


def softmax_attention(q, k, v, talk, scale, window, keep, rows=slice(None)):
    """The queries ``rows`` of a whole sequence; float64.  q [T, H, P], k and v [T, G, .]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    per = H // G
    q = q[rows]
    scores = torch.stack([q[:, h] @ k[:, h // per].T for h in range(H)]) * scale
    if talk is not None:
        scores = plain.mix_scores(scores, talk)
    weights = torch.softmax(scores.masked_fill(~plain.visible(T, window, keep)[rows], -float("inf")), dim=-1)
    return torch.stack([weights[h] @ v[:, h // per] for h in range(H)], dim=1)


def designed(T, H, G, P, V, window, keep, at, td, seed=0):
    """Queries, keys, values and a mixing matrix: weak random keys, and for the query at position ``at`` strong ones at both
    edges of its window and of the kept tokens; values name their position."""
    g = torch.Generator().manual_seed(seed)
    q = torch.randn(T, H, P, generator=g) * 0.3
    k = torch.randn(T, G, P, generator=g) * 0.3
    v = torch.randn(T, G, V, generator=g)
    talk = torch.randn(H, H, generator=g) * 0.3 + 0.5 * torch.eye(H)
    direction = torch.randn(P, generator=g)
    q[at] = direction * 0.5 + 0.1 * q[at]
    talk[talk.sum(dim=1) < 0.2] += 0.4  # every head's mixed score rises with a key along the direction
    for j in {at, at - window + 1, at - window, keep - 1, keep, 0} if window else {at, 0, at // 2}:
        if 0 <= j <= at:
            k[j] = direction * 0.5
            v[j] = v[j].sign() * (1.0 + j / 37.0)
    td_round = lambda t: t.to(td).float()
    return td_round(q), td_round(k), td_round(v), talk


SIZES = [  # H, G, P, V, window, keep, page size
    (4, 2, 64, 64, 40, 5, 16), (8, 8, 64, 24, 64, 64, 8), (16, 4, 128, 128, 100, 1, 16), (6, 1, 128, 96, 129, 140, 32),
    (16, 1, 64, 64, 1, 17, 16), (32, 8, 128, 128, 70, 30, 64), (12, 3, 128, 33, 33, 0, 16), (20, 10, 64, 64, 250, 20, 128),
    (5, 5, 64, 48, None, 0, 16), (24, 2, 64, 64, 128, 128, 8), (64, 8, 128, 128, 60, 25, 16)]


@pytest.mark.parametrize("H,G,P,V,window,keep,page_size", SIZES)
@pytest.mark.parametrize("mixed", [True, False])
def test_attention_on_designed_keys(H, G, P, V, window, keep, page_size, mixed):
    """The one-warp-a-row kernel in both types, the prompt kernel over a portion, the single-token kernel alone and with its
    keys shared among several CTAs; every page no query of the step can see is page 0, which is full of NaN."""
    from torchlet_b200 import ops

    T, first, scale = 421, 300, 0.31
    for at in (420, 383, 331):
        for dtype in DTYPES:
            td = TORCH[dtype]
            q, k, v, talk = designed(T, H, G, P, V, window, keep, at, td, seed=at)
            if not mixed:
                talk = None
            padded_v = torch.cat([v, torch.zeros(T, G, P - V)], dim=2)
            exact = lambda window, keep, rows: softmax_attention(q.double(), k.double(), v.double(), talk.double() if mixed else None,
                                                                 scale, window, keep, rows)
            want = exact(window, keep, slice(first, None))
            if window:  # a mask that is one token off must show
                for w2, k2 in ((window + 1, keep), (window - 1, keep), (window, keep + 1), (window, max(0, keep - 1))):
                    off = exact(max(1, w2), k2, slice(at, at + 1))[0]
                    if not torch.equal(plain.visible(T, max(1, w2), k2)[at], plain.visible(T, window, keep)[at]):
                        assert (off - want[at - first]).abs().max() > 0.15 * want[at - first].abs().max()
            pages, table = _paged(k, padded_v, page_size, td, seed=at)

            def tables(pos):
                """The block table of a step whose first new token is at ``pos``: pages given back are page 0."""
                out = table.clone()
                if window:
                    gone = max(0, pos - window + 1) // page_size
                    out[:, -(-keep // page_size):gone] = 0
                return out

            rows = (spread(q.double(), talk.double(), G) if mixed else q.double()[:, :, None]).reshape(T, -1).to(td).to(DEV)
            n = T - first
            common = dict(nh=H, nkv=G, p_size=P, page_size=page_size, window=window, keep=keep, v_cols=V, scale=scale)
            got = torch.full((n, H * V), float("nan"), dtype=td, device=DEV)
            part = rows[first:].contiguous()
            ops.attention_generic(part, part.stride(0), pages, tables(first), i32([0] * n), i32(range(first, T)), got, n, H, G, P,
                                  page_size, window, scale, keep=keep, spread=mixed, v_cols=V)
            tol = 5e-5 if dtype == "float32" else 3e-2
            close(got.view(n, H, V)[at - first], want[at - first], tol, f"one warp a row, {dtype}, the designed query")
            close(got.view(n, H, V), want, tol, f"one warp a row, {dtype}")
            if dtype == "float32":
                continue
            got.fill_(float("nan"))
            per_tile = ops.attention_spread_rows(H // G)
            starts = list(range(0, n * (H // G), per_tile))
            ops.attention_spread(part, pages, tables(first), i32([0, n]), i32([first]), i32([0] * len(starts)), i32(starts),
                                 len(starts), got, spread=mixed, **common)
            close(got.view(n, H, V)[at - first], want[at - first], tol, "prompt kernel, the designed query")
            close(got.view(n, H, V), want, tol, "prompt kernel")
            assert ops.attention_spread_error() == 0
            if not ops.attention_mixed_decode_tile(H, G, P, page_size, V):
                assert H // G > 16 or H > 64
                continue
            one = q[at].reshape(1, -1).to(td).to(DEV)
            for splits in (1, 2, 7, 40):
                got = torch.full((1, H * V), float("nan"), dtype=td, device=DEV)
                ops.attention_mixed_decode(one, pages, tables(at), i32([0, 1]), i32([at]), None, 1, got,
                                           talk=talk.to(DEV) if mixed else None, splits=splits, **common)
                close(got.view(H, V), want[at - first], tol, f"single token, {splits} splits")
            assert ops.attention_mixed_decode_error() == 0


def test_single_tokens_of_several_requests_beside_one_another():
    """Requests of very different lengths in one launch, a few of them, not all of the step's."""
    from torchlet_b200 import ops

    H, G, P, window, keep, page_size, scale = 8, 2, 64, 50, 10, 16, 0.3
    td = torch.bfloat16
    lengths = [1, 3, 200, 65, 128, 11]
    pool, tables, want, queries = [], torch.zeros(len(lengths), 16, dtype=torch.int32), [], []
    talk = rand(H, H, seed=2, scale=0.5)
    for r, n in enumerate(lengths):
        q, k, v = (rand(n, heads, P, seed=10 * r + s).to(td).float() for s, heads in ((1, H), (2, G), (3, G)))
        pages, table = _paged(k, v, page_size, td, seed=r)
        base = sum(p.shape[0] for p in pool)
        tables[r, :table.shape[1]] = table[0].cpu() + base
        pool.append(pages)
        queries.append(q[-1].reshape(-1))
        want.append(softmax_attention(q.double(), k.double(), v.double(), talk.double(), scale, window, keep)[-1])
    chosen = [0, 2, 3, 5]
    q = torch.stack(queries).to(td).to(DEV)
    for splits in (1, 3):
        out = torch.full((len(lengths), H * P), 7.0, dtype=td, device=DEV)
        ops.attention_mixed_decode(q, torch.cat(pool), tables.to(DEV), i32(range(len(lengths) + 1)), i32([n - 1 for n in lengths]),
                                   i32(chosen), len(chosen), out, nh=H, nkv=G, p_size=P, page_size=page_size, window=window,
                                   keep=keep, v_cols=P, scale=scale, talk=talk.to(DEV), splits=splits)
        for r in range(len(lengths)):
            if r in chosen:
                close(out[r].view(H, P), want[r], 3e-2, f"request {r}, {splits} splits")
            else:
                assert (out[r] == 7.0).all()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_kept_key_among_thousands(dtype):
    """5,000 cached tokens; the one key that stands out is the last kept token, far before the window."""
    from torchlet_b200 import ops

    H, G, P, window, keep, page_size, T, scale = 4, 2, 64, 300, 21, 16, 5000, 0.3
    td = TORCH[dtype]
    k, v = rand(T, G, P, seed=1, scale=0.2).to(td).float(), rand(T, G, P, seed=2, scale=0.1).to(td).float()
    direction = rand(P, seed=3).to(td).float()
    k[keep - 1], k[keep] = direction, direction
    v[keep - 1], v[keep] = 1.0, -1.0
    talk = torch.eye(H) * 0.7 + 0.1
    q = direction.repeat(H, 1)[None]
    pages, table = _paged(k, v, page_size, td, seed=4)
    table[:, 2:(T - window) // page_size] = 0
    rows = spread(q.double(), talk.double(), G).reshape(1, -1).to(td).to(DEV)
    got = torch.empty(1, H * P, dtype=td, device=DEV)
    ops.attention_generic(rows, rows.stride(0), pages, table, i32([0]), i32([T - 1]), got, 1, H, G, P, page_size, window, scale,
                          keep=keep, spread=True, v_cols=P)
    assert (got.float() - 1).abs().max() < 0.02
    if dtype == "bfloat16":
        for splits in (1, 6):
            got.zero_()
            ops.attention_mixed_decode(q.reshape(1, -1).to(td).to(DEV), pages, table, i32([0, 1]), i32([T - 1]), None, 1, got,
                                       nh=H, nkv=G, p_size=P, page_size=page_size, window=window, keep=keep, v_cols=P,
                                       scale=scale, talk=talk.to(DEV), splits=splits)
            assert (got.float() - 1).abs().max() < 0.02


# ------------------------------------------------------------------ between product and attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V,P,dims", [(4, 2, 24, 16, 64, 8), (6, 6, 10, 18, 64, 10), (16, 4, 128, 128, 128, 128),
                                            (9, 3, 64, 20, 64, 32), (17, 1, 16, 64, 64, 0), (8, 1, 136, 30, 136, 40)])
@pytest.mark.parametrize("mode", ["spread", "plain", "by request", "unmixed"])
def test_norm_rotation_value_mixing_and_cache_rows(dtype, H, G, D, V, P, dims, mode):
    """Split sums with a bias and finished rows, two requests (one brings a single token) behind cached tokens, far into a
    sequence; the kernel's split-half rotation of reordered rows against the interleaved one."""
    from torchlet_b200 import ops
    from torchlet_b200.parts.rotary import pair_permutation

    td, eps, page_size, base = TORCH[dtype], 1e-3, 16, 300.0
    lengths, before = [5, 1, 3], [0, 1000, 37]
    positions = [b + i for n, b in zip(lengths, before) for i in range(n)]
    req = [r for r, n in enumerate(lengths) for _ in range(n)]
    T, width = len(positions), H * D + G * (D + V)
    proj, bias = rand(T, width, seed=1), rand(width, seed=2)
    wq, wk, talk = 1 + rand(H * D, seed=3, scale=0.2), 1 + rand(G * D, seed=4, scale=0.2), rand(H, H, seed=5, scale=0.5)
    first, lam = rand(T, G * V, seed=6), torch.tensor([0.3])
    x = (proj + bias).double()
    q = plain.rms_norm(x[:, :H * D], wq.double(), eps).view(T, H, D)
    k = plain.rms_norm(x[:, H * D:(H + G) * D], wk.double(), eps).view(T, G, D)
    if dims:
        pos = torch.tensor(positions, dtype=torch.float64)
        q, k = plain.rotate_pairs(q, pos, base, dims), plain.rotate_pairs(k, pos, base, dims)
    own = x[:, (H + G) * D:]
    mixed = plain.mix_values(own, first.double(), lam.double())

    order = pair_permutation(D, dims, "interleaved")
    reorder = lambda t, heads: t.reshape(*t.shape[:-1], heads, D)[..., order].reshape(*t.shape[:-1], heads * D)
    laid = lambda t: torch.cat([reorder(t[..., :H * D], H), reorder(t[..., H * D:(H + G) * D], G), t[..., (H + G) * D:]], dim=-1)
    inv = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float32).to(DEV) if dims else None
    want_q = torch.cat([q[..., order], torch.zeros(T, H, P - D)], dim=2)
    want_spread = spread(want_q, talk.double(), G).reshape(T, -1)
    tol = 3e-5 if dtype == "float32" else 6e-3
    form = {"spread": 1, "plain": 0, "by request": 2, "unmixed": 1}[mode]
    for splits, value_mode in ((None, 0), (None, 1), (3, 2)):
        pages = torch.zeros(80, 2, G, page_size, P, dtype=td, device=DEV)
        table = torch.arange(1, 79, dtype=torch.int32).view(1, -1).repeat(3, 1)
        table[1], table[2] = torch.roll(table[1], 7), torch.roll(table[2], 20)
        if splits:
            parts = torch.stack([laid(proj) * f for f in (0.5, 0.2, 0.3)]).to(DEV)
            source = dict(src=parts, splits=3, row=width, bias=laid(bias).to(DEV))
        else:
            source = dict(src=laid(proj + bias).to(DEV))
        values = first.clone().to(DEV)
        out = torch.full((T, H * P * G), float("nan"), dtype=td, device=DEV)
        ops.qkv_prepare(sizes=(H, G, D, V, P), positions=i32(positions), token_req=i32(req), req_indptr=i32([0, 5, 6, 9]),
                        block_table=table.to(DEV), pages=pages, page_size=page_size, q_out=out, wq=reorder(wq, H).to(DEV),
                        wk=reorder(wk, G).to(DEV), eps=eps, inv_freq=inv, mix=None if mode == "unmixed" else talk.to(DEV),
                        spread=form, v_first=values if value_mode else None, value_lambda=lam.to(DEV) if value_mode == 2 else None,
                        **source)
        for t in range(T):
            as_spread = mode == "spread" or (mode == "by request" and lengths[req[t]] > 1)
            got = out[t] if as_spread else out[t, :H * P]
            close(got, want_spread[t] if as_spread else want_q[t].reshape(-1), tol, f"queries of token {t}")
            page = int(table[req[t], positions[t] // page_size])
            close(pages[page, 0, :, positions[t] % page_size, :D], k[t][:, order], tol, f"keys of token {t}")
            want_v = (mixed if value_mode == 2 else own)[t].view(G, V)
            close(pages[page, 1, :, positions[t] % page_size, :V], want_v, tol, f"values of token {t}")
            assert (pages[page, 0, :, positions[t] % page_size, D:] == 0).all()
            assert (pages[page, 1, :, positions[t] % page_size, V:] == 0).all()
        if value_mode == 1:
            close(values, own, 1e-5, "values left to later layers")
        elif value_mode == 2:
            assert torch.equal(values.cpu(), first)
        assert int((pages != 0).any(dim=(1, 2, 4)).sum()) <= T, "no other row is touched"


# ------------------------------------------------------------------ token pairs
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,streams,buckets,mul_prev,mul_cur", [(44, 1, 1, 3, 11), (96, 3, 37, 5, 3), (300, 2, 991, 31, 7),
                                                                     (64, 5, 50, 10 ** 12 + 39, 10 ** 11 + 3)])
@pytest.mark.parametrize("norm", ["layer", "rms", None])
def test_token_pairs_across_steps_slots_and_padding(dtype, width, streams, buckets, mul_prev, mul_cur, norm):
    """Two requests in portions (one of them a single token at a time) and a padding lane; a third then takes the first one's
    slot: its first token must not see the token the slot still holds."""
    from torchlet_b200 import ops

    td, vocab, eps, scale = TORCH[dtype], 61, 1e-4, 1.5
    table, pairs = rand(vocab, width, seed=1).to(td), rand(buckets + 1, width, seed=2).to(td)
    w, b = 1 + rand(width, seed=3, scale=0.2), rand(width, seed=4, scale=0.3)
    last = torch.tensor([11, 12, 13, 14], dtype=torch.int32, device=DEV)
    g = torch.Generator().manual_seed(5)
    seqs = [torch.randint(0, vocab, (n,), generator=g).tolist() for n in (19, 12, 6)]

    def want(ids):
        rows = plain.bigram_rows(ids, buckets, mul_prev, mul_cur)
        x = table.double()[ids] * scale + pairs.double()[rows]
        if norm == "layer":
            x = plain.layer_norm(x, w.double(), eps) + b.double()
        elif norm == "rms":
            x = plain.rms_norm(x, w.double(), eps)
        return x[:, None].expand(-1, streams, -1)

    def step(lengths, before, slots, ids):
        indptr = [0]
        for n in lengths:
            indptr.append(indptr[-1] + n)
        out = torch.full((indptr[-1], streams, width), float("nan"), device=DEV)
        ops.token_embed(table.to(DEV), i32(ids), out, scale=scale, pairs=(pairs.to(DEV), mul_prev, mul_cur),
                        norm={"layer": (w.to(DEV), b.to(DEV), eps, True), "rms": (w.to(DEV), None, eps, False), None: None}[norm],
                        ctx_arrays=(i32([b0 + i for n, b0 in zip(lengths, before) for i in range(n)]),
                                    i32([r for r, n in enumerate(lengths) for _ in range(n)]), i32(indptr), i32(slots)), last=last)
        return out

    at, got = [0, 0], [[], []]
    for n0, n1 in ((7, 1), (2, 1), (1, 5), (1, 1), (8, 4)):
        ids = seqs[0][at[0]:at[0] + n0] + seqs[1][at[1]:at[1] + n1] + [0]
        out = step([n0, n1, 1], [at[0], at[1], 0], [2, 0, -1], ids)  # the last lane is padding
        got[0].append(out[:n0])
        got[1].append(out[n0:n0 + n1])
        at = [at[0] + n0, at[1] + n1]
        assert last.tolist() == [seqs[1][at[1] - 1], 12, seqs[0][at[0] - 1], 14]
    close(torch.cat(got[0]), want(seqs[0]), 1e-5, "request 0")
    close(torch.cat(got[1]), want(seqs[1]), 1e-5, "request 1")
    close(torch.cat([step([2], [0], [2], seqs[2][:2]), step([4], [2], [2], seqs[2][2:])]), want(seqs[2]), 1e-5, "a slot used again")


# ------------------------------------------------------------------ routed ungated experts
def test_router_bias_and_softmax_over_the_chosen_logits():
    from torchlet_b200 import ops

    logits = torch.tensor([[0.0, 5.0, 4.0, 0.1, 4.5, 0.2], [1.0, 1.0, 1.0, 1.0, 1.0, 1.0], [300.0, 299.0, -300.0, 0.0, 298.5, 1.0],
                           [-90.0, -91.0, -90.5, -200.0, -200.0, -200.0]])
    x, router = torch.eye(4, 8), torch.zeros(6, 8)
    router[:, :4] = logits.T
    for bias in (torch.zeros(6), torch.tensor([4.8, 0.0, -1.0, 0.0, 0.3, 2.0])):  # the second one changes choices
        for top in (1, 2, 4, 6):
            choice = torch.empty(4, top, dtype=torch.int32, device=DEV)
            weight = torch.empty(4, top, device=DEV)
            ops.moe_route(x.to(DEV), router.to(DEV), choice, weight, bias=bias.to(DEV), chosen_softmax=True)
            z = logits.double() + bias.double()
            for t in range(4):
                want = sorted(range(6), key=lambda e: (-float(z[t, e]), e))[:top]
                assert choice[t].cpu().tolist() == want
                close(weight[t], torch.softmax(z[t, want], dim=0), 1e-6, f"weights of token {t}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,top,width,ff,tokens", [(6, 2, 96, 40, 150), (1, 1, 64, 24, 7), (3, 3, 64, 24, 33), (8, 2, 128, 64, 300),
                                                   (16, 4, 128, 64, 1), (4, 1, 50, 21, 70), (12, 3, 256, 320, 600),
                                                   (32, 2, 64, 48, 20), (5, 2, 44, 12, 3)])
def test_routed_ungated_experts(dtype, E, top, width, ff, tokens):
    """The whole part on inputs that both sides hold exactly, without close calls of the router."""
    from torchlet_b200.config.spec import PartSpec
    from torchlet_b200.parts import FEED_FORWARDS, build_part

    td = TORCH[dtype]
    rounded = lambda *shape, seed, scale: rand(*shape, seed=seed, scale=scale).to(torch.bfloat16).float()
    w = {"router": rounded(E, width, seed=E, scale=0.15), "router.b": rounded(E, seed=E + 1, scale=0.5)}
    for e in range(E):
        w[f"e{e}.up"] = rounded(ff, width, seed=40 + e, scale=0.3)
        w[f"e{e}.down"] = rounded(width, ff, seed=70 + e, scale=0.3)
    x = rand(tokens + 20, width, seed=21, scale=1.2).to(td).float()
    z = (x.double() @ w["router"].double().T + w["router.b"].double()).sort(dim=1, descending=True).values
    if E > 1:
        x = x[(z[:, :-1] - z[:, 1:]).amin(dim=1) > 1e-4]
    x = x[:tokens]
    mlp = {"router": {"experts": E, "top": top}, "expert": {"ff": ff}}
    want = plain.mixture({"m." + k: v.double() for k, v in w.items()}, "m.", mlp, x.double())
    part = build_part(FEED_FORWARDS, PartSpec("routed_clamped_glu", {
        "hidden_size": width, "intermediate_size": ff, "unit": "relu_squared", "num_experts": E, "top_k": top,
        "score": "chosen_softmax", "router_bias": True, "weight_on": "output"}))
    part.load({"m." + k: v for k, v in w.items()}, "m.", DEV, td)
    ctx = Ctx(td, [x.shape[0]], [0], [0])
    acc = torch.zeros(x.shape[0], width, device=DEV)
    part.forward(ctx, x.to(td).to(DEV), acc)
    close(acc, want, 3e-5 if dtype == "float32" else 2e-2, "routed ungated experts")
