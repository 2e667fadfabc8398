"""Each mechanism of the Tekarax design alone: the kernels and parts against the plain functions of
tests/plain_tekarax.py, at sizes of their own, with inputs designed so that a fault shows (sinks that outweigh every key,
keys just inside and just outside a window, one far key whose value must arrive turned by its distance, stale pages full
of NaN, states and last rows that must carry over portions, slots and hundreds of steps, gates and biases that count)."""
import pytest
import torch

import plain_tekarax as plain
from test_kilatar_parts_gpu import DEV, TORCH, Cache, Ctx, _paged, close, no_deferred_sums, rand

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


def bf16(w):
    return {k: t.to(torch.bfloat16).float() for k, t in w.items()}


def double(w):
    return {k: t.double() for k, t in w.items()}


def host_planned(ctx, lengths, before):
    """What parts that plan on the host read of a step."""
    ctx.req_indptr_host, ctx.kv_before_host = ctx.req_indptr.cpu().numpy(), ctx.kv_before.cpu().numpy()
    ctx.max_kv_len = max(b + n for b, n in zip(before, lengths))
    ctx.max_q_len = max(lengths)
    ctx.upload = lambda values: torch.as_tensor(values, dtype=torch.int32).to(DEV)
    return ctx


# ------------------------------------------------------------------ learned sinks
SINKS = torch.tensor([-4.0, 0.0, 3.0, 9.0, 1.0, -1.0])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [None, 17])
def test_learned_sink_of_the_plain_kernel(dtype, window):
    """Heads whose sink is lost in the sum, level with the keys, and outweighs all of them by far."""
    from torchlet_b200 import ops

    H, G, d, T, scale, page_size, td = 6, 2, 24, 130, 0.4, 8, TORCH[dtype]
    k, v, q = (rand(T, n, d, seed=s).to(td).float() for n, s in ((G, 1), (G, 2), (H, 3)))
    want = plain.softmax_attention(q.double(), k.double(), v.double(), scale, window=window, sink=SINKS.double())
    pages, table = _paged(k, v, page_size, td, seed=3)
    out = torch.full((T, H * d), float("nan"), dtype=td, device=DEV)
    i32 = lambda t: t.to(torch.int32).to(DEV)
    ops.attention_generic(q.reshape(T, H * d).to(td).to(DEV), H * d, pages, table, i32(torch.zeros(T)), i32(torch.arange(T)),
                          out, T, H, G, d, page_size, window, scale, sink=SINKS.to(DEV))
    for h in range(H):  # head by head: the head of the largest sink has the smallest output
        close(out.view(T, H, d)[:, h], want[:, h], 3e-5 if dtype == "float32" else 2e-2, f"head {h}")


@pytest.mark.parametrize("d,H,G", [(64, 6, 1), (128, 6, 2), (64, 6, 6)])
@pytest.mark.parametrize("window,page_size", [(None, 16), (150, 8)])
def test_learned_sink_of_the_tensor_core_kernels(d, H, G, window, page_size):
    """Portions on mma.sync and tcgen05 (whole, with key splits, with the merge deferred) and single tokens with the key
    splits merged inside the kernel and by the second kernel, against the one-warp-a-row kernel on the same pages."""
    from torchlet_b200 import ops

    T, scale, g, td, sink = 500, d ** -0.5, H // G, torch.bfloat16, SINKS.to(DEV)
    k, v, q = (rand(T, n, d, seed=s) for n, s in ((G, 21), (G, 22), (H, 23)))
    pages, table = _paged(k, v, page_size, td, seed=d)
    qd = q.reshape(T, H * d).to(td).to(DEV)
    pos = torch.arange(T, dtype=torch.int32, device=DEV)
    zeros = torch.zeros(T, dtype=torch.int32, device=DEV)
    want = torch.empty(T, H * d, dtype=td, device=DEV)
    ops.attention_generic(qd, H * d, pages, table, zeros, pos, want, T, H, G, d, page_size, window, scale, sink=sink)
    indptr = torch.tensor([0, T], dtype=torch.int32, device=DEV)
    before = torch.zeros(1, dtype=torch.int32, device=DEV)

    def check(got, rows, what):
        for h in range(H):
            close(got.view(-1, H, d)[:, h], want.view(T, H, d)[rows, h].float().cpu(), 2e-2, f"{what}, head {h}")

    rows = torch.arange(0, T * g, 64, dtype=torch.int32, device=DEV)
    got = torch.full((T, H * d), float("nan"), dtype=td, device=DEV)
    ops.attention_mma(qd, pages, table, indptr, before, torch.zeros_like(rows), rows, rows.numel(), got, T, H, G, d, page_size,
                      window, scale, rows16=False, sink=sink)
    check(got, slice(None), "portion")
    rows = torch.arange(0, T * g, ops.attention_tc_rows(g), dtype=torch.int32, device=DEV)
    for splits, defer in ((1, False), (3, False), (2, True)):
        got = torch.full((T, H * d), float("nan"), dtype=td, device=DEV)
        merge = ops.attention_tc(qd, pages, table, indptr, before, torch.zeros_like(rows), rows, rows.numel(), got, H, G, d,
                                 page_size, window, scale, splits=splits, token_req=zeros, defer_merge=defer, sink=sink)
        if defer:
            merge()
        check(got, slice(None), f"portion on tcgen05, {splits} key splits")
    ops.raise_on_wait_errors()
    for at in (T - 1, 0, 64):
        indptr = torch.tensor([0, 1], dtype=torch.int32, device=DEV)
        before = torch.tensor([at], dtype=torch.int32, device=DEV)
        for splits in (1, 3, 20):
            one = torch.full((1, H * d), float("nan"), dtype=td, device=DEV)
            ops.attention_mma(qd[at:at + 1], pages, table, indptr, before, None, None, 1, one, 1, H, G, d, page_size, window,
                              scale, rows16=True, splits=splits, sink=sink)
            check(one, slice(at, at + 1), f"single token at {at}, {splits} key splits")


# ------------------------------------------------------------------ turned values, one gate a head
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nh,d,vdim,gated", [(3, 24, 24, True), (2, 24, 10, True), (5, 64, 64, True), (1, 128, 96, False),
                                             (2, 40, 0, True), (4, 16, 16, False)])
def test_outputs_turn_back_and_take_one_gate_a_head(dtype, nh, d, vdim, gated):
    from torchlet_b200 import ops

    td, T = TORCH[dtype], 9
    o = rand(T, nh, d, seed=nh).to(td).float()
    pos = torch.tensor([0, 1, 2, 63, 64, 999, 4000, 17, 5])
    freq = plain.plain_frequencies(500.0, vdim) if vdim else None
    gate = rand(T, 2 + nh, seed=7, scale=2.0)
    want = plain.rotate_halves(o.double(), -pos, freq) if vdim else o.double()
    if gated:
        want = want * torch.sigmoid(gate[:, 2:].double())[:, :, None]
    rows = o.reshape(T, nh * d).to(td).to(DEV)
    ops.head_finish(rows, pos.to(torch.int32).to(DEV), freq.float().to(DEV) if vdim else None,
                    gate.to(DEV)[:, 2:] if gated else None, nh, d)
    close(rows.view(T, nh, d), want, 3e-4 if dtype == "float32" else 1e-2, "finished heads")


ATTENTION_SIZES = [(4, 2, 24, 16, 8), (2, 2, 8, 20, 4), (3, 1, 40, 40, 40), (4, 1, 64, 64, 32), (2, 1, 64, 128, 64), (8, 4, 128, 128, 128)]


def _attention_part(m, width, td, w):
    from torchlet_b200.config import PartSpec
    from torchlet_b200.parts import MIXERS, build_part

    rot = m["rot"]
    part = build_part(MIXERS, PartSpec("gated_attention", {
        "hidden_size": width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_dim": m["vdim"],
        "scale": m["scale"], "sink": "learned", "gate": "head_sigmoid", "eps": 1e-6,
        "positions": PartSpec("rotary_partial", {"head_dim": m["dim"], "dims": rot["dims"], "base": rot["base"], "scaling": rot.get("scaling")}),
        "value_rotation": PartSpec("rotary_partial", {"head_dim": m["vdim"], "dims": m["vdim"], "base": rot["base"]})}))
    part.load(w, "a.", DEV, td)
    no_deferred_sums(part)
    return part


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V,dims", ATTENTION_SIZES)
def test_attention_mixer_with_turned_values(dtype, H, G, D, V, dims):
    """The mixer alone, as a whole prompt, and as portions and single tokens.  The last query and one key 250 positions
    back stand out on an entry that does not turn (or turns slowest): the value it fetches must arrive turned by the
    distance; its head's sink and gate must count."""
    td, width, T, page = TORCH[dtype], 64, 290, 16
    m = {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": 0.21,
         "rot": {"base": 30000.0, "dims": dims, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64}}}
    w = {"a.q": rand(H * D, width, seed=1, scale=0.2), "a.k": rand(G * D, width, seed=2, scale=0.2),
         "a.v": rand(G * V, width, seed=3, scale=0.3), "a.g": rand(H, width, seed=6, scale=0.3),
         "a.sink": rand(H, seed=7, scale=1.5), "a.o": rand(width, H * V, seed=4, scale=0.3)}
    still = D - 1 if dims < D else dims // 2 - 1
    h = rand(T, width, seed=5)
    h[:, 9] = 0.0
    h[T - 1, 9] = h[39, 9] = 4.0
    w["a.q"].view(H, D, width)[:, still, 9] = 2.5
    w["a.k"].view(G, D, width)[:, still, 9] = 2.5
    w, h = bf16(w), h.to(td).float()
    want = plain.attention(m, double(w), "a.", h.double())
    part = _attention_part(m, width, td, w)
    P = part.kv_spec().head_dim
    pages = torch.full((40, 2, G, page, P), float("nan"), dtype=td, device=DEV)
    table = (torch.randperm(39, generator=torch.Generator().manual_seed(3))[:20] + 1).to(torch.int32).view(1, -1).to(DEV)

    def run(n, before):
        cache = Cache(None)
        cache.pages, cache.block_table, cache.page_size = pages, table, page
        acc = torch.zeros(n, width, device=DEV)
        part.forward(host_planned(Ctx(td, [n], [before], [0]), [n], [before]), h[before:before + n].to(td).to(DEV), acc, cache)
        return acc

    tol = 5e-5 if dtype == "float32" else 3e-2
    whole = run(T, 0)
    close(whole, want, tol, "whole prompt")
    close(whole[T - 1], want[T - 1], tol, "the far key's value")
    pages.fill_(float("nan"))
    got = torch.cat([run(70, 0), run(2, 70), run(198, 72)] + [run(1, t) for t in range(270, T)])
    close(got, want, tol, "portions and single tokens")
    close(got[T - 1], want[T - 1], tol, "the far key's value, decoded")
    w["a.sink"] = w["a.sink"] + 8.0  # the plain functions with this far larger sink differ: the test sees a lost sink
    assert (plain.attention(m, double(w), "a.", h.double()) - want).abs().max() > 0.2 * want.abs().max()


# ------------------------------------------------------------------ latent attention over a window
LATENT_SIZES = [(3, 20, 28, 40), (1, 8, 8, 16), (4, 32, 32, 64), (2, 24, 16, 130), (8, 48, 32, 256), (70, 8, 8, 32)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,V,rank", LATENT_SIZES)
@pytest.mark.parametrize("size", [1, 7, 64, 100, 1000])
def test_latent_attention_over_a_window(dtype, H, D, V, rank, size):
    """No positions at all.  For the last query the key just INSIDE its window and the key just OUTSIDE stand out; pages
    that only hold keys before every window are NaN again when the single tokens run, as after being given back."""
    from torchlet_b200.config import PartSpec
    from torchlet_b200.parts import MIXERS, build_part

    td, width, eps, T, page = TORCH[dtype], 64, 1e-5, 300, 16
    m = {"heads": H, "dim": D, "vdim": V, "kv_rank": rank, "scale": 0.3, "mask": {"size": size}}
    w = {"l.q": rand(H * D, width, seed=1, scale=0.2), "l.dkv": rand(rank, width, seed=2, scale=0.2),
         "l.dkv.norm": 1.0 + rand(rank, seed=3, scale=0.2), "l.uk": rand(H * D, rank, seed=4, scale=0.2),
         "l.uv": rand(H * V, rank, seed=5, scale=0.2), "l.o": rand(width, H * V, seed=7, scale=0.3)}
    h = rand(T, width, seed=8)
    last = T - 1
    for j, at in enumerate(a for a in (last - size + 1, last - size) if 0 <= a < last):
        h[at, 5 + j] += 8.0
    w = bf16(w)
    # the queries of the last token look for the two latents' directions
    c = plain.rms(h.double() @ w["l.dkv"].double().T, eps) * w["l.dkv.norm"].double()
    for at in (last - size + 1, last - size):
        if 0 <= at < last:
            aim = (c[at] @ w["l.uk"].double().T).view(H, D)
            h[last] += 0.4 * (torch.linalg.pinv(w["l.q"].double()) @ aim.reshape(-1)).float()
    h = h.to(td).float()
    want = plain.latent_attention(m, double(w), "l.", h.double(), eps)
    part = build_part(MIXERS, PartSpec("latent_attention", {
        "hidden_size": width, "num_heads": H, "head_dim": D, "rot_dim": 0, "v_dim": V, "q_rank": None, "kv_rank": rank,
        "scale": 0.3, "eps": eps, "window": size}))
    part.load(w, "l.", DEV, td)
    no_deferred_sums(part)
    assert part.kv_spec().group_key() == (1, rank, size, 1)
    pages = torch.full((40, page, rank), float("nan"), dtype=td, device=DEV)
    table = (torch.randperm(39, generator=torch.Generator().manual_seed(5))[:20] + 1).to(torch.int32).view(1, -1).to(DEV)

    def run(n, before):
        cache = Cache(None)
        cache.pages, cache.block_table, cache.page_size = pages, table, page
        acc = torch.zeros(n, width, device=DEV)
        part.forward(host_planned(Ctx(td, [n], [before], [0]), [n], [before]), h[before:before + n].to(td).to(DEV), acc, cache)
        for p in range(max(0, before + n - size) // page):  # passed pages change hands
            pages[int(table[0, p])] = float("nan")
        return acc

    tol = 5e-5 if dtype == "float32" else 4e-2
    whole = run(T, 0)
    close(whole, want, tol, "whole prompt")
    close(whole[last], want[last], tol, "the window's edge")
    pages.fill_(float("nan"))
    got = torch.cat([run(130, 0), run(2, 130), run(158, 132)] + [run(1, t) for t in range(290, T)])
    close(got, want, tol, "portions and single tokens")
    close(got[last], want[last], tol, "the window's edge, decoded")


def test_window_splits_of_single_tokens_equal_one_cta():
    """One token behind 1,999 cached rows under windows of several sizes, its keys over 1, 2, 5 and 40 CTAs."""
    from torchlet_b200 import ops

    H, dk, T, page, td = 5, 64, 2000, 16, torch.bfloat16
    rows = rand(T, 1, dk, seed=1)
    pages = torch.full((140, page, dk), float("nan"), dtype=td, device=DEV)
    table = (torch.randperm(139, generator=torch.Generator().manual_seed(6))[:125] + 1).to(torch.int32).view(1, -1)
    for t in range(T):
        pages[int(table[0, t // page]), t % page] = rows[t, 0].to(td)
    q = rand(1, H * dk, seed=2, scale=0.7).to(td).to(DEV)
    i32 = lambda *v: torch.tensor(v, dtype=torch.int32, device=DEV)
    table = table.to(DEV)
    for window in (None, 1, 63, 64, 65, 700, 1999, 2500):
        want = torch.empty(1, H * dk, dtype=td, device=DEV)
        ops.latent_attention(q, pages, table, i32(0), i32(T - 1), want, 1, H, dk, dk, page, 0.2, window=window)
        for splits in (1, 2, 5, 40):
            got = torch.full((1, H * dk), float("nan"), dtype=td, device=DEV)
            ops.latent_attention_mma(q, pages, table, i32(0, 1), i32(T - 1), None, None, 1, got, 1, H, dk, dk, page, 0.2, splits,
                                     window=window)
            close(got, want.float().cpu(), 2e-2, f"window {window}, {splits} splits")


# ------------------------------------------------------------------ token shift and time mixing
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,n", [(96, 5), (50, 3), (513, 1), (2048, 5)])
def test_token_shift_over_portions_slots_and_padding(dtype, width, n):
    from torchlet_b200 import ops

    td = TORCH[dtype]
    seqs = [rand(k, width, seed=i).to(td).float() for i, k in enumerate((23, 9))]
    mu = rand(n, width, seed=9)
    wants = [torch.stack([plain.token_shift(s.double(), mu[c].double()) for c in range(n)]) for s in seqs]
    state = torch.zeros(4, width, device=DEV)
    state[3] = float("nan")
    at, got = [0, 0], [[], []]
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
    for a, b in ((1, 2), (10, 1), (2, 1), (1, 1), (9, 4)):
        x = torch.cat([seqs[0][at[0]:at[0] + a], seqs[1][at[1]:at[1] + b], torch.ones(1, width)]).to(td).to(DEV)
        out = torch.full((n, a + b + 6, width), float("nan"), dtype=td, device=DEV)
        ops.token_shift(x, mu.to(DEV), out, state, i32([0] * a + [1] * b + [2]), i32([0, a, a + b, a + b + 1]), i32([2, 0, -1]), 3)
        got[0].append(out[:, :a].cpu())
        got[1].append(out[:, a:a + b].cpu())
        close(out[:, a + b], (torch.ones(n, width) - mu).double(), 1e-2 if dtype == "bfloat16" else 1e-6, "padding: zeros before it")
        at = [at[0] + a, at[1] + b]
    for r in range(2):
        close(torch.cat(got[r], dim=1), wants[r], 1e-2 if dtype == "bfloat16" else 1e-6, f"request {r}")
    assert torch.isnan(state[3]).all() and float(state[1].abs().max()) == 0.0
    assert torch.equal(state[2].cpu(), seqs[0][-1]) and torch.equal(state[0].cpu(), seqs[1][-1])


def _mixing_weights(H, D, rank, width, seed):
    w = {f"t.mu.{c}": 0.5 + rand(width, seed=seed + i, scale=0.3) for i, c in enumerate("rkvgw")}
    w.update({f"t.{c}": rand(H * D, width, seed=seed + 10 + i, scale=0.3) for i, c in enumerate("rkvg")})
    w.update({"t.w1": rand(rank, width, seed=seed + 20, scale=0.3), "t.w2": rand(H * D, rank, seed=seed + 21, scale=0.5),
              "t.w0": -1.5 + rand(H * D, seed=seed + 22), "t.u": rand(H, D, seed=seed + 23),
              "t.norm": 1.0 + rand(H * D, seed=seed + 24, scale=0.3), "t.o": rand(width, H * D, seed=seed + 25, scale=0.3)})
    return bf16(w)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,rank,width", [(3, 12, 7, 48), (1, 8, 1, 64), (2, 64, 24, 64), (1, 128, 16, 40), (1, 250, 9, 32), (5, 10, 3, 50)])
def test_time_mixing_carries_state_and_last_row(dtype, H, D, rank, width):
    """Two requests of unequal length in portions down to ONE and two tokens beside a padding lane; the second request then
    runs again in the slot the first one left (cleared), and a NaN slot nobody owns stays NaN."""
    from torchlet_b200.config import PartSpec
    from torchlet_b200.parts import MIXERS, build_part

    td, eps = TORCH[dtype], 1e-5
    m, w = {"heads": H, "dim": D}, _mixing_weights(H, D, rank, width, seed=H + D)
    part = build_part(MIXERS, PartSpec("time_mixing", {"hidden_size": width, "num_heads": H, "head_dim": D, "decay_rank": rank, "eps": eps}))
    part.load(w, "t.", DEV, td)
    no_deferred_sums(part)
    seqs = [rand(n, width, seed=30 + i).to(td).float() for i, n in enumerate((57, 23))]
    wants = [plain.wkv(m, double(w), "t.", s.double(), eps) for s in seqs]
    state = {name: torch.zeros((4, *spec.slot_shape(512)), device=DEV) for name, spec in part.state_spec().items()}
    for t in state.values():
        t[3] = float("nan")  # nobody's slot
    cuts = [[7, 1, 2, 30, 1, 1, 15], [2, 1, 9, 1, 3, 6, 1]]
    at, got = [0, 0], [[], []]
    for step in range(7):
        lengths = [cuts[0][step], cuts[1][step], 1]  # the third lane is padding (slot -1)
        ctx = Ctx(td, lengths, [at[0], at[1], 0], [0, 2, -1])
        x = torch.cat([seqs[0][at[0]:at[0] + lengths[0]], seqs[1][at[1]:at[1] + lengths[1]], torch.ones(1, width)])
        acc = torch.zeros(sum(lengths), width, device=DEV)
        part.forward(ctx, x.to(td).to(DEV), acc, Cache(state))
        got[0].append(acc[:lengths[0]].cpu())
        got[1].append(acc[lengths[0]:lengths[0] + lengths[1]].cpu())
        at = [at[0] + lengths[0], at[1] + lengths[1]]
    # a head's norm divides by what may be near zero at the first tokens: bfloat16 is judged behind them
    skip, tol = (0, 1e-4) if dtype == "float32" else (4, 8e-2)
    for r in range(2):
        close(torch.cat(got[r])[skip:], wants[r][skip:], tol, f"request {r}")
    for t in state.values():
        assert torch.isnan(t[3]).all() and torch.isfinite(t[:3]).all() and float(t[1].abs().max()) == 0.0
        t[0].zero_()  # admission clears the slot
    acc = torch.zeros(23, width, device=DEV)
    part.forward(Ctx(td, [23], [0], [0]), seqs[1].to(td).to(DEV), acc, Cache(state))
    close(acc[skip:], wants[1][skip:], tol, "in a slot used again")


@pytest.mark.parametrize("tokens", [1, 3, 8, 16, 17, 40, 130, 300])
def test_time_mixing_products_at_many_token_counts(tokens):
    """Sizes the tensor cores take, at token counts on both sides of every choice of the products' kernels: one token a
    request (the recurrences stand alone) against the 32-bit path."""
    from torchlet_b200.config import PartSpec
    from torchlet_b200.parts import MIXERS, build_part

    H, D, rank, width, eps = 2, 64, 24, 192, 1e-5
    w = _mixing_weights(H, D, rank, width, seed=3)
    h = rand(tokens, width, seed=1).to(torch.bfloat16).float()
    outs = []
    for td in (torch.float32, torch.bfloat16):
        part = build_part(MIXERS, PartSpec("time_mixing", {"hidden_size": width, "num_heads": H, "head_dim": D, "decay_rank": rank, "eps": eps}))
        part.load(w, "t.", DEV, td)
        no_deferred_sums(part)
        g = torch.Generator().manual_seed(9)
        state = {n: torch.randn((tokens, *s.slot_shape(64)), generator=g).to(DEV) for n, s in part.state_spec().items()}
        acc = torch.zeros(tokens, width, device=DEV)
        part.forward(Ctx(td, [1] * tokens, [0] * tokens, range(tokens), capacity=300), h.to(td).to(DEV), acc, Cache(state))
        outs.append((acc.cpu(), state["matrix"].cpu()))
    close(outs[1][0], outs[0][0].double(), 3e-2, "outputs")
    close(outs[1][1], outs[0][1].double(), 3e-2, "states")


@pytest.mark.parametrize("H,D,rank,width", [(3, 16, 5, 64), (2, 20, 40, 72), (4, 32, 1, 64), (2, 64, 24, 128), (1, 96, 70, 64),
                                            (3, 128, 200, 128), (2, 100, 100, 64)])
@pytest.mark.parametrize("tokens", [1, 5, 16, 20, 40, 64])
def test_single_tokens_in_one_kernel_walk_on_as_the_portions_do(H, D, rank, width, tokens):
    """Many requests, one token each, four steps in a row from states that a portion has left, every third lane padding,
    slots in a scrambled order: the stacked products and the one-kernel step against the plain recurrence."""
    from torchlet_b200 import ops
    from torchlet_b200.config import PartSpec
    from torchlet_b200.parts import MIXERS, build_part

    td, eps, steps = torch.bfloat16, 1e-5, 4
    m, w = {"heads": H, "dim": D}, _mixing_weights(H, D, rank, width, seed=D)
    part = build_part(MIXERS, PartSpec("time_mixing", {"hidden_size": width, "num_heads": H, "head_dim": D, "decay_rank": rank, "eps": eps}))
    part.load(w, "t.", DEV, td)
    no_deferred_sums(part)
    assert part.one_kernel
    slots = torch.randperm(tokens + 2, generator=torch.Generator().manual_seed(tokens))[:tokens].tolist()
    slots = [-1 if i % 3 == 2 else s for i, s in enumerate(slots)]
    live = [i for i, s in enumerate(slots) if s >= 0]
    state = {name: torch.full((tokens + 2, *spec.slot_shape(64)), float("nan"), device=DEV) for name, spec in part.state_spec().items()}
    for t in state.values():
        for i in live:
            t[slots[i]] = 0.0
    seqs = {i: rand(6 + steps, width, seed=100 + i).to(td).float() for i in live}
    for i in live:  # six tokens as a portion
        part.forward(Ctx(td, [6], [0], [slots[i]], capacity=512), seqs[i][:6].to(td).to(DEV), torch.zeros(6, width, device=DEV), Cache(state))
    calls, inner = [], ops.time_mixing_step
    ops.time_mixing_step = lambda *a, **k: (calls.append(1), inner(*a, **k))
    try:
        got = []
        for k in range(steps):
            x = torch.stack([seqs[i][6 + k] if i in seqs else torch.ones(width) for i in range(tokens)])
            acc = torch.zeros(tokens, width, device=DEV)
            part.forward(Ctx(td, [1] * tokens, [6 + k] * tokens, slots, capacity=512), x.to(td).to(DEV), acc, Cache(state))
            got.append(acc.cpu())
            for i in range(tokens):
                if slots[i] < 0:
                    assert float(acc[i].abs().max()) == 0.0
    finally:
        ops.time_mixing_step = inner
    assert len(calls) == steps
    for i in live[:: max(1, len(live) // 6)]:
        want = plain.wkv(m, double(w), "t.", seqs[i].double(), eps)[6:]
        close(torch.stack([g[i] for g in got]), want, 6e-2, f"request {i}")
    for t in state.values():  # slots nobody owns are as they were
        owned = {slots[i] for i in live}
        assert all(bool(torch.isnan(t[s]).all()) == (s not in owned) for s in range(tokens + 2))


def test_the_bonus_meets_the_current_token_only_and_the_state_remembers():
    """A decay near one keeps the first token's value for 600 tokens, through portions and single tokens; the bonus shows
    in a token's own output and never in the state."""
    from torchlet_b200 import ops

    H, D, T = 1, 8, 600
    r, k, v = torch.zeros(T, D), torch.zeros(T, D), torch.zeros(T, D)
    k[0, 0], v[0] = 1.0, torch.arange(1, D + 1).float()
    r[0, 0] = r[T - 1, 0] = 1.0
    planes = torch.stack([r, k, v]).to(DEV)
    decay = torch.full((T, D), 0.9999, device=DEV)
    bonus = torch.full((H, D), 2.5, device=DEV)
    state = torch.zeros(2, H, D, D, device=DEV)
    out = torch.empty(T, D, device=DEV)
    at = 0
    for n in [1, 200, 1, 1, 396, 1]:
        cut = planes[:, at:at + n].contiguous()
        ops.gla_scan(cut[0], decay[at:at + n].contiguous(), torch.tensor([0, n], dtype=torch.int32, device=DEV),
                     torch.tensor([1], dtype=torch.int32, device=DEV), state, out[at:at + n], 1, H, D, D, 1.0,
                     bonus=bonus, k_offset=n * D, v_offset=2 * n * D)
        at += n
    close(out[0], 2.5 * torch.arange(1, D + 1).double(), 1e-6, "the token's own bonus")
    close(out[T - 1], torch.arange(1, D + 1).double() * 0.9999 ** (T - 2), 1e-5, "remembered without the bonus")
    assert float(out[1:T - 1].abs().max()) == 0.0 and float(state[0].abs().max()) == 0.0


@pytest.mark.parametrize("H,D", [(2, 12), (1, 33), (3, 64), (1, 200)])
def test_scan_with_bonus_against_the_plain_recurrence(H, D):
    from torchlet_b200 import ops

    T = 37
    r, k, v = (rand(T, H, D, seed=s) for s in (1, 2, 3))
    decay, u = torch.sigmoid(rand(T, H, D, seed=4, scale=2.0)), rand(H, D, seed=5)
    want = plain.wkv_scan(r.double(), k.double(), v.double(), decay.double(), u.double())
    planes = torch.stack([r, k, v]).reshape(3, T, H * D).contiguous().to(DEV)
    state = torch.zeros(1, H, D, D, device=DEV)
    out = torch.empty(T, H * D, device=DEV)
    ops.gla_scan(planes[0], decay.reshape(T, H * D).contiguous().to(DEV), torch.tensor([0, T], dtype=torch.int32, device=DEV),
                 torch.zeros(1, dtype=torch.int32, device=DEV), state, out, 1, H, D, D, 1.0, bonus=u.to(DEV),
                 k_offset=T * H * D, v_offset=2 * T * H * D)
    close(out.view(T, H, D), want, 2e-5, "scan")


@pytest.mark.parametrize("tokens,channels,rank", [(1, 36, 7), (19, 130, 1), (8, 300, 64)])
def test_decay_of_a_tanh_through_two_exponentials(tokens, channels, rank):
    """w0 from far below (decay one) to far above (decay zero): nothing overflows on the way."""
    from torchlet_b200 import ops

    low, w2 = rand(tokens, rank + 3, seed=1, scale=2.0), rand(channels, rank, seed=2)
    w0 = torch.linspace(-30.0, 30.0, channels)
    z = torch.tanh(low[:, 3:].double()) @ w2.double().T + w0.double()
    out = torch.empty(tokens, channels, device=DEV)
    ops.gla_decay(low.to(DEV), 3, w2.t().contiguous().to(DEV), w0.to(DEV), out, rank, 0.0)
    got = out.cpu().double()
    want = torch.exp(-torch.exp(z))
    assert torch.isfinite(got).all() and float((got - want).abs().max()) < 2e-6
    assert float(got.max()) == 1.0 and float(got.min()) == 0.0


# ------------------------------------------------------------------ the end of a sub-layer
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [50, 96, 1024, 1100, 2048, 4100, 9000])
@pytest.mark.parametrize("centre,splits,gate_splits,row,following",
                         [(True, 0, 0, False, True), (True, 3, 2, True, True), (False, 5, 1, True, False), (True, 0, 4, False, False),
                          (False, 1, 0, False, True)])
def test_norm_behind_a_sublayer_with_gate_sums_and_the_next_norm(dtype, width, centre, splits, gate_splits, row, following):
    from torchlet_b200 import ops

    T, eps, m, td = 5, 1e-5, 0.7, TORCH[dtype]
    acc, y = rand(T, width, seed=1), rand(T, width, seed=2) + 3.0
    y[1] = 0.0  # a row that is all but constant: eps counts
    parts, gates = rand(max(splits, 1), T, width, seed=3), rand(max(gate_splits, 1), T, width, seed=4)
    parts[:, 1] *= 1e-3
    yb, gb, weight, bias, step, w2 = (rand(width, seed=s) for s in (5, 6, 7, 8, 9, 10))
    yb[:] *= 1e-3
    v = y.double() + (parts.double().sum(0) if splits else 0.0) + yb.double()
    if gate_splits:
        v = v * torch.sigmoid(gates.double().sum(0) + gb.double())
    norm = lambda x, w: plain.layer_norm(x, w, eps) if centre else plain.rms(x, eps) * w
    want = acc.double() + m * (norm(v, weight.double()) + bias.double()) + (step.double() if row else 0.0)
    dev = lambda t: t.contiguous().to(DEV)
    a, side = dev(acc), dev(y)
    out = torch.full((T, width), float("nan"), dtype=td, device=DEV) if following else None
    ops.residual_norm(a, side, dev(weight), eps, bias=dev(bias), centre=centre, m=m, partials=dev(parts) if splits else None,
                      splits=splits, y_bias=dev(yb), gate=dev(gates) if gate_splits else None, gate_splits=gate_splits,
                      gate_bias=dev(gb) if gate_splits else None, row=dev(step) if row else None, clear=True,
                      following=(dev(w2), None, eps, True, out) if following else None)
    close(a, want, 2e-5, "stream")
    assert float(side.abs().max()) == 0.0
    if following:
        close(out, plain.layer_norm(want, w2.double(), eps), 5e-5 if dtype == "float32" else 1e-2, "the next norm")


def test_a_row_is_added_to_every_token():
    from torchlet_b200 import ops

    for T, width in ((1, 50), (7, 96), (300, 2048)):
        acc, row = rand(T, width, seed=1), rand(width, seed=2)
        a = acc.to(DEV)
        ops.add_row(a, row.to(DEV))
        assert torch.equal(a.cpu(), acc + row)


@pytest.mark.parametrize("gated", [True, False])
def test_an_rms_norm_behind_a_gated_sublayer_keeps_its_own_path_without_a_gate(gated):
    """``add_normed`` of an RMS norm with a gate goes through the same pending sum as a layer norm's."""
    from torchlet_b200.config import PartSpec
    from torchlet_b200.engine.runner import StepContext
    from torchlet_b200.parts import NORMS, build_part

    T, width, eps = 3, 40, 1e-6
    norm = build_part(NORMS, PartSpec("rms_norm", {"size": width, "eps": eps}))
    weight = rand(width, seed=1)
    norm.load({"n.weight": weight}, "n.", DEV, torch.float32)

    class Runner:
        dtype, device, token_capacity = torch.float32, DEV, 8

        def buffer(self, name, shape, dtype):
            return torch.empty(shape, dtype=dtype, device=DEV)

    ctx = StepContext(Runner())
    acc, y, g = rand(T, width, seed=2), rand(T, width, seed=3), rand(T, width, seed=4)
    a, side = acc.to(DEV), y.to(DEV)
    norm.add_normed(ctx, side, a, clear=True, **({"gate": (g.to(DEV), 0, None)} if gated else {}))
    x = norm.apply(ctx, a)
    v = y.double() * (torch.sigmoid(g.double()) if gated else 1.0)
    want = acc.double() + plain.rms(v, eps) * weight.double()
    close(a, want, 1e-5, "stream")
    close(x, plain.rms(want, eps) * weight.double(), 1e-5, "next norm")
    assert float(side.abs().max()) == 0.0


# ------------------------------------------------------------------ feed-forwards
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,ff,tokens", [(96, 40, 33), (64, 72, 1), (128, 192, 300), (50, 21, 17), (256, 512, 8), (512, 2048, 130)])
def test_ungated_unit_with_squared_relu_and_biases(dtype, width, ff, tokens):
    from torchlet_b200.config import PartSpec
    from torchlet_b200.parts import FEED_FORWARDS, build_part

    td = TORCH[dtype]
    w = bf16({"f.up": rand(ff, width, seed=2, scale=width ** -0.5), "f.down": rand(width, ff, seed=3, scale=0.3),
              "f.up.b": rand(ff, seed=5), "f.down.b": rand(width, seed=6)})
    x = rand(tokens, width, seed=7, scale=1.5).to(td).float()
    want = plain.dense_unit(double(w), "f.", x.double())
    part = build_part(FEED_FORWARDS, PartSpec("mlp", {"hidden_size": width, "intermediate_size": ff, "bias": True}))
    part.load(w, "f.", DEV, td)
    no_deferred_sums(part)
    acc = torch.zeros(tokens, width, device=DEV)
    part.forward(Ctx(td, [tokens], [0], [0]), x.to(td).to(DEV), acc)
    close(acc, want, 2e-5 if dtype == "float32" else 3e-2, "ungated unit")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,top,width,ff,shared,tokens", [(6, 2, 96, 24, 40, 150), (1, 1, 64, 24, 16, 40), (3, 3, 64, 24, 0, 33),
                                                          (8, 2, 128, 64, 64, 500), (12, 1, 256, 96, 96, 1), (5, 4, 50, 21, 13, 70)])
def test_experts_whose_sigmoid_weights_multiply_their_inputs_beside_a_shared_one(dtype, E, top, width, ff, shared, tokens):
    """The whole part on inputs that both sides hold exactly, with close calls of the choice taken out.  Under silu a weight
    on the input differs from one on the output; the shared expert has no gate and no weight."""
    from torchlet_b200.config import PartSpec
    from torchlet_b200.parts import FEED_FORWARDS, build_part

    td = TORCH[dtype]
    w = {"m.router": rand(E, width, seed=E, scale=0.15)}
    for e in list(range(E)):
        w.update({f"m.e{e}.{n}": rand(*((width, ff) if n == "down" else (ff, width)), seed=10 * e + i, scale=0.3)
                  for i, n in enumerate(("gate", "up", "down"))})
    if shared:
        w.update({f"m.shared.{n}": rand(*((width, shared) if n == "down" else (shared, width)), seed=500 + i, scale=0.3)
                  for i, n in enumerate(("gate", "up", "down"))})
    w = bf16(w)
    x = rand(tokens, width, seed=20, scale=1.2).to(td).float()
    ranked = torch.sigmoid(x.double() @ w["m.router"].double().T).sort(dim=1, descending=True).values
    if top < E and tokens > 1:
        x = x[(ranked[:, :top] - ranked[:, 1:top + 1]).amin(dim=1) > 1e-4]
        tokens = x.shape[0]
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": E, "top": top}, **({"shared": {"ff": shared}} if shared else {})}
    want = plain.mixture(mlp, double(w), "m.", x.double())
    chosen, weights = plain.route(mlp, double(w), "m.", x.double())
    part = build_part(FEED_FORWARDS, PartSpec("routed_clamped_glu", {
        "hidden_size": width, "intermediate_size": ff, "limit": None, "num_experts": E, "top_k": top, "score": "sigmoid",
        "renormalize": False, "weight_on": "input", "shared_prefix": "shared.",
        "shared": PartSpec("gated_mlp", {"hidden_size": width, "intermediate_size": shared, "activation": "silu", "bias": False}) if shared else None}))
    part.load(w, "m.", DEV, td)
    if part.shared is not None:
        no_deferred_sums(part.shared)
    ctx = Ctx(td, [tokens], [0], [0])
    acc = torch.zeros(tokens, width, device=DEV)
    part.forward(ctx, x.to(td).to(DEV), acc)
    close(acc, want, 3e-5 if dtype == "float32" else 3e-2, "routed experts")
    assert torch.equal(ctx.buffers[("moe.choice", (top,), torch.int32)][:tokens].cpu().long(), chosen)
    close(ctx.buffers[("moe.weight", (top,), torch.float32)][:tokens], weights, 1e-5, "weights")
