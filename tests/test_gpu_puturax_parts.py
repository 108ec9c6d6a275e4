"""The kernels behind the Puturax mechanisms, each alone against the plain evaluation (``plain_puturax.py``) of the same inputs:
biased and squashed attention over shuffled pages (row-wise and in the prompt kernel, a far key that stands out, page borders,
poisoned unused rows), the preparation of queries, keys and values, the router's choice, mixtures of neighbouring tokens, the
recurrence in order, in chunks, in pieces and token by token, products of several mixtures in one launch, and the norm on a
sublayer's output with the norm that follows it."""

import math

import pytest
import torch

import plain_puturax as P

pytestmark = pytest.mark.gpu

F = torch.float64
DEV = "cuda"


def K():
    from dryft_b200.ops import kernels

    return kernels


def rel(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return float((got - want).abs().max() / want.abs().max().clamp(min=1e-30))


class Ctx:
    """The step's metadata of sequences that each bring some tokens behind some earlier ones."""

    def __init__(self, lens, starts=None, slots=None, tile=64):
        starts = starts or [0] * len(lens)
        slots = slots if slots is not None else list(range(len(lens)))[::-1]
        cu = [0]
        for n in lens:
            cu.append(cu[-1] + n)
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
        self.n_seqs, self.cu_q, self.seq_slot = len(lens), i32(cu), i32(slots)
        self.tok_slot = i32([s for s, n in zip(slots, lens) for _ in range(n)])
        self.tok_pos = i32([st + j for st, n in zip(starts, lens) for j in range(n)])
        tiles = [(c + q, min(tile, n - q)) for c, n in zip(cu, lens) for q in range(0, n, tile)]
        self.tile_tok0, self.tile_rows, self.n_tiles, self.tile_size = i32([t[0] for t in tiles]), i32([t[1] for t in tiles]), len(tiles), tile
        self.bounds = list(zip(cu, cu[1:]))


# ----------------------------------------------------------------------------- biased attention
def _paged(rows, slots, page, dtype, seed):
    """Rows ``[L, G, D]`` of each sequence in pages at shuffled places; what no row fills is NaN."""
    g = torch.Generator().manual_seed(seed)
    need = [(r.shape[0] + page - 1) // page for r in rows]
    order = torch.randperm(sum(need) + 3, generator=g).tolist()
    G, D = rows[0].shape[1:]
    pages = torch.full((sum(need) + 3, G, page, D), float("nan"), dtype=dtype)
    table = torch.zeros((max(slots) + 1, max(need) + 1), dtype=torch.int32)
    at = 0
    for r, s, n in zip(rows, slots, need):
        for p in range(n):
            table[s, p] = order[at]
            part = r[p * page:(p + 1) * page]
            pages[order[at], :, :part.shape[0]] = part.transpose(0, 1).to(dtype)
            at += 1
    return pages.to(DEV), table.to(DEV)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, G, D, DV, cap, bias, form", [
    (4, 2, 16, 16, 6.0, True, "both"), (3, 3, 32, 48, None, True, "both"), (6, 2, 48, 16, 25.0, False, "both"), (4, 1, 10, 21, 3.0, True, "rows"),
    (2, 1, 64, 64, 12.0, True, "both")])
def test_biased_and_squashed_attention(dtype, H, G, D, DV, cap, bias, form):
    g = torch.Generator().manual_seed(H * 100 + D)
    lens, slots = [1, 63, 64, 65, 300], [4, 0, 2, 5, 1]
    r1, r2 = torch.rand(H, generator=g) * 1.5, torch.rand(H, generator=g) * 0.5 + 0.01
    scale = 1.7 / math.sqrt(D)
    qs, ks, vs = ([torch.randn(n, h, d, generator=g) for n in lens] for h, d in ((H, D), (G, D), (G, DV)))
    # far keys, and keys on both sides of a page's edge, that single queries ask for: their scores stand out by several units
    for i, j in ((299, 0), (299, 63), (298, 64), (200, 5), (129, 127), (128, 128), (64, 63)):
        for h in range(H):
            ks[4][j, h // (H // G)] += 0.5 * qs[4][i, h]
    qs, ks, vs = ([t.to(dtype).float() for t in ts] for ts in (qs, ks, vs))
    want = []
    for q, k, v in zip(qs, ks, vs):
        o = torch.empty(q.shape[0], H, DV, dtype=F)
        for h in range(H):
            s = P.squash((q[:, h].double() @ k[:, h // (H // G)].double().T) * scale, cap)
            if bias:
                s = s - P.distance_bias(q.shape[0], float(r1[h]), float(r2[h]))
            o[:, h] = P.weights_of(s, True) @ v[:, h // (H // G)].double()
        want.append(o)
    want = torch.cat(want)
    ctx = Ctx(lens, slots=slots)
    kp, table = _paged(ks, slots, 64, dtype, 1)
    vp, _ = _paged(vs, slots, 64, dtype, 1)
    q = torch.cat(qs).to(dtype).to(DEV)
    n = q.shape[0]
    one = torch.zeros(H, device=DEV)
    kw = dict(softcap=cap, dist_bias=(r1.to(DEV), r2.to(DEV)) if bias else None)
    tol = 2e-5 if dtype == torch.float32 else 1.5e-2
    for splits in (1, 5):
        out = torch.empty((n, H, DV), dtype=dtype, device=DEV)
        po, pml = torch.empty((n, H, splits, DV), device=DEV), torch.empty((n, H, splits, 2), device=DEV)
        K().pool_attn_rows(q, kp, vp, table, None, one, ctx.tok_slot, ctx.tok_pos, out, scale, 1 << 30, 0, splits, po, pml, **kw)
        assert rel(out, want) <= tol, f"rows, {splits} splits"
    if dtype == torch.bfloat16 and form == "both":
        out = torch.empty((n, H, DV), dtype=dtype, device=DEV)
        K().pool_attn_prefill(q, kp, vp, table, None, one, ctx.tile_tok0, ctx.tile_rows, ctx.tok_slot, ctx.tok_pos, out, ctx.n_tiles, scale, 1 << 30, 0, **kw)
        assert rel(out, want) <= tol, "prompt kernel"
        # a piece behind an earlier one: tiles that start anywhere, seen through the same pages
        piece = Ctx([300 - 171], starts=[171], slots=[1])
        part = torch.empty((129, H, DV), dtype=dtype, device=DEV)
        K().pool_attn_prefill(q[-129:].contiguous(), kp, vp, table, None, one, piece.tile_tok0, piece.tile_rows, piece.tok_slot, piece.tok_pos, part,
                              piece.n_tiles, scale, 1 << 30, 0, **kw)
        assert rel(part, want[-129:]) <= tol, "prompt kernel, a piece"


def test_squashed_scores_of_any_size_stay_finite():
    """Scores of hundreds of caps either way: the squashed score is the cap, the softmax that of equal scores."""
    H, D = 2, 16
    for sign in (1.0, -1.0):
        q = torch.full((70, H, D), 60.0, dtype=torch.bfloat16, device=DEV)
        k = torch.full((70, H, D), 60.0 * sign)
        v = torch.randn(70, H, D, generator=torch.Generator().manual_seed(0))
        kp, table = _paged([k], [0], 64, torch.bfloat16, 0)
        vp, _ = _paged([v], [0], 64, torch.bfloat16, 0)
        ctx = Ctx([70])
        out = torch.empty((70, H, D), dtype=torch.bfloat16, device=DEV)
        K().pool_attn_prefill(q, kp, vp, table, None, None, ctx.tile_tok0, ctx.tile_rows, ctx.tok_slot, ctx.tok_pos, out, ctx.n_tiles, 1.0, 1 << 30, 0, softcap=4.0)
        want = torch.cumsum(v.to(torch.bfloat16).double(), 0) / torch.arange(1, 71, dtype=F)[:, None, None]
        assert rel(out, want) <= 2e-2


def test_refused_combinations():
    from dryft_b200.ops.kernels import KernelError

    x = torch.zeros((1, 2, 16), dtype=torch.bfloat16, device=DEV)
    pages = torch.zeros((1, 2, 64, 16), dtype=torch.bfloat16, device=DEV)
    i = torch.zeros((1, 1), dtype=torch.int32, device=DEV)
    with pytest.raises(KernelError, match="pooled"):
        K().pool_attn_rows(x, pages, pages, i, (pages, pages, i), None, i[0], i[0], x.clone(), 1.0, 8, 4, softcap=2.0)
    with pytest.raises(KernelError, match="positive cap"):
        K().pool_attn_rows(x, pages, pages, i, None, None, i[0], i[0], x.clone(), 1.0, 8, 0, softcap=-2.0)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, G, D, DV, qt", [(4, 2, 16, 24, (0.6, 7)), (3, 1, 70, 33, (0.25, 1)), (2, 2, 8, 130, None)])
def test_preparation_of_queries_keys_and_values(dtype, H, G, D, DV, qt):
    g = torch.Generator().manual_seed(D)
    lens, starts = [1, 90, 130], [0, 55, 3]
    ctx = Ctx(lens, starts)
    n, eps = sum(lens), 1e-3
    proj = (torch.randn(n, H * D + G * (D + DV) + 5, generator=g) * 0.3).to(dtype)
    slots = ctx.seq_slot.tolist()
    table = torch.zeros((3, 4), dtype=torch.int32)
    table.view(-1)[torch.randperm(12, generator=g)] = torch.arange(12, dtype=torch.int32)
    kp, vp = torch.full((12, G, 64, D), 9.0, dtype=dtype, device=DEV), torch.full((12, G, 64, DV), 9.0, dtype=dtype, device=DEV)
    q = torch.empty((n, H, D), dtype=dtype, device=DEV)
    K().pool_attn_prep(proj.to(DEV), None, None, None, None, None, 0, ctx.tok_slot, ctx.tok_pos, q, kp, vp, table.to(DEV), H, G, eps, True, v_eps=eps, q_temp=qt)
    x = proj.double()
    temp = P.temperature(200, {"coef": qt[0], "every": qt[1]} if qt else None)[ctx.tok_pos.cpu().long()]
    wq = P.unit_rms(x[:, :H * D].view(n, H, D), eps) * temp[:, None, None]
    wk = P.unit_rms(x[:, H * D:(H + G) * D].view(n, G, D), eps)
    wv = P.unit_rms(x[:, (H + G) * D:(H + G) * D + G * DV].view(n, G, DV), eps)
    tol = 2e-6 if dtype == torch.float32 else 5e-3
    assert rel(q, wq) <= tol
    pos, tab = ctx.tok_pos.tolist(), table.tolist()
    at = [(tab[s][p // 64], p % 64) for s, p in zip(ctx.tok_slot.tolist(), pos)]
    assert slots == [2, 1, 0]
    assert rel(torch.stack([kp[a, :, b] for a, b in at]), wk) <= tol and rel(torch.stack([vp[a, :, b] for a, b in at]), wv) <= tol
    assert int((vp != 9.0).any(-1).sum()) == n * G                 # nothing else was written


# ----------------------------------------------------------------------------- the router
@pytest.mark.parametrize("E, top, groups, corr", [(8, 3, (2, 1), -0.4), (8, 3, (4, 2), 0.0), (6, 2, None, -2.0), (12, 4, (12, 5), -1.0), (1, 1, None, 0.3),
                                                  (96, 7, (8, 3), -0.6), (6, 6, (3, 3), 0.1)])
def test_choices_with_corrections_and_groups(E, top, groups, corr):
    g = torch.Generator().manual_seed(E + top)
    n, width = 40, 64
    h, w = torch.randn(n, width, generator=g), torch.randn(E, width, generator=g) * 0.4
    c = corr + torch.randn(E, generator=g) * 0.3
    router = {"experts": E, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    idx, wts = P.router_choice(h.double(), router, {"router": w.double(), "correction": c.double()}, "")
    cnt, keep = groups or (1, 1)
    kw = dict(renorm=True, score="sigmoid", correction=c.to(DEV), group_rank="top2", renorm_eps=1e-20)
    for rows in (False, True):
        gi, gw = torch.empty((n, top), dtype=torch.int32, device=DEV), torch.empty((n, top), device=DEV)
        if rows:
            K().moe_route_rows(h.to(DEV), w.to(DEV), cnt, keep, top, gi, gw, **kw)
        else:
            K().moe_route((h @ w.T).to(DEV), cnt, keep, top, gi, gw, **kw)
        assert torch.equal(gi.cpu().long(), idx) and float((gw.cpu().double() - wts).abs().max()) < 1e-5


def test_tiny_scores_are_divided_by_more_than_their_sum():
    z = torch.tensor([[-60.0, -70.0, -47.0]], device=DEV)
    idx, wts = torch.empty((1, 2), dtype=torch.int32, device=DEV), torch.empty((1, 2), device=DEV)
    K().moe_route(z, 1, 1, 2, idx, wts, renorm=True, score="sigmoid", correction=torch.zeros(3, device=DEV), group_rank="top2", renorm_eps=1e-20)
    s = torch.sigmoid(z.double().cpu())[0][[2, 0]]
    assert idx[0].tolist() == [2, 0] and torch.allclose(wts[0].double().cpu(), s / (s.sum() + 1e-20), rtol=1e-4)
    assert float(wts.sum()) < 0.5          # the sum was below the number that joins it


# ----------------------------------------------------------------------------- time mixing
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [64, 37])
def test_mixtures_of_a_token_and_the_one_before(dtype, width):
    g = torch.Generator().manual_seed(width)
    ctx = Ctx([1, 5, 2, 9], slots=[3, 0, 2, 5])
    h, last, mu = torch.randn(17, width, generator=g).to(dtype), torch.randn(6, width, generator=g).to(dtype), torch.rand(5, width, generator=g)
    out = torch.empty((5, 17, width), dtype=dtype, device=DEV)
    K().wkv_mix(h.to(DEV), last.to(DEV), mu.to(DEV), ctx.tok_slot, out)
    prev = torch.cat([torch.cat([last[s][None], h[a:b - 1]]) for s, (a, b) in zip((3, 0, 2, 5), ctx.bounds)]).double()
    want = torch.stack([h.double() + (prev - h.double()) * mu[j].double() for j in range(5)])
    assert rel(out, want) <= (1e-6 if dtype == torch.float32 else 5e-3)


def _wkv(H, d, lens, dtype, seed, strong):
    g = torch.Generator().manual_seed(seed)
    n = sum(lens)
    t = {k: torch.randn(n, H * d, generator=g).to(dtype) for k in "rkvg"}
    # decays from exp(-20) to 1 - 1e-4 side by side, or of ordinary strength
    t["z"] = torch.randn(n, H * d, generator=g) * (2.0 if strong else 0.5)
    t["w0"] = (torch.rand(H * d, generator=g) * 12.0 - 9.0) if strong else torch.full((H * d,), -2.0)
    t["u"], t["norm"] = torch.randn(H * d, generator=g), 1.0 + 0.3 * torch.randn(H * d, generator=g)
    t["h"] = torch.randn(n, 24, generator=g).to(dtype)
    return t


def _wkv_plain(t, H, d, bounds, eps):
    outs, states = [], []
    for a, b in bounds:
        f = lambda k: t[k][a:b].double().view(b - a, H, d)
        w = torch.exp(-torch.exp(f("z") + t["w0"].double().view(H, d)))
        o = torch.stack([P.decayed_outer_products(f("r")[:, i], f("k")[:, i], f("v")[:, i], w[:, i], t["u"].double().view(H, d)[i]) for i in range(H)], 1)
        outs.append((P.unit_rms(o, eps) * t["norm"].double().view(H, d) * P.silu(f("g"))).reshape(b - a, H * d))
        S = torch.zeros(H, d, d, dtype=F)
        for s in range(b - a):
            S = w[s][:, :, None] * S + f("k")[s][:, :, None] * f("v")[s][:, None, :]
        states.append(S)
    return torch.cat(outs), states


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, d, strong", [(3, 16, False), (2, 5, True), (2, 40, True), (2, 64, True), (1, 100, False), (1, 200, True), (1, 30, False)])
def test_the_recurrence_in_order_in_chunks_and_in_pieces(dtype, H, d, strong):
    lens, slots, eps = [300, 1, 64, 129, 2], [2, 0, 5, 1, 3], 1e-5
    t = _wkv(H, d, lens, dtype, d, strong)
    ctx = Ctx(lens, slots=slots)
    want, states = _wkv_plain(t, H, d, ctx.bounds, eps)
    g = {k: v.to(DEV) for k, v in t.items()}
    tol = 3e-5 if dtype == torch.float32 else 6e-3
    n = sum(lens)

    def run(parts, chunked):
        """Every sequence cut at the same fractions; the pieces of all of them are one step."""
        state = torch.full((6, H, d, d), float("nan"), device=DEV)
        last = torch.full((6, 24), float("nan"), dtype=dtype, device=DEV)
        state[slots], last[slots] = 0.0, 0.0
        out = torch.empty((n, H * d), dtype=dtype, device=DEV)
        for f0, f1 in parts:
            rows, piece, sl = [], [], []
            for s, (a, b) in zip(slots, ctx.bounds):
                lo, hi = a + int((b - a) * f0), a + int((b - a) * f1)
                if hi > lo:
                    rows += list(range(lo, hi))
                    piece.append(hi - lo)
                    sl.append(s)
            c = Ctx(piece, slots=sl)
            sub = {k: g[k][rows].contiguous() for k in ("r", "k", "v", "g", "z", "h")}
            o = torch.empty((len(rows), H * d), dtype=dtype, device=DEV)
            K().wkv_tokens(sub["r"], sub["k"], sub["v"], sub["g"], sub["z"], g["w0"], g["u"], g["norm"], eps, sub["h"], last, c, state, o, chunked=chunked)
            out[rows] = o
        return out, state, last

    for parts, chunked in (([(0, 1)], False), ([(0, 1)], True), ([(0, 0.3), (0.3, 0.31), (0.31, 1)], True), ([(0, 0.5), (0.5, 1)], False)):
        out, state, last = run(parts, chunked)
        what = f"{len(parts)} pieces, chunked {chunked}"
        assert rel(out, want) <= tol, what
        for s, S, (a, b) in zip(slots, states, ctx.bounds):
            assert rel(state[s], S) <= (2e-5 if dtype == torch.float32 else 1e-4), what
            assert torch.equal(last[s], g["h"][b - 1]), what


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, d, R, strong", [(3, 16, 5, False), (2, 5, 1, True), (2, 64, 16, True), (1, 200, 24, True), (2, 130, 40, False), (1, 300, 8, False)])
def test_the_recurrence_token_by_token(dtype, H, d, R, strong):
    """One launch a token with the decay's second product inside, for sequences side by side and padding between them; against
    the walk of the same tokens."""
    eps, L, slots = 1e-5, 12, [4, -1, 1]
    t = _wkv(H, d, [L, L], dtype, d, strong)
    gen = torch.Generator().manual_seed(5)
    low, w2 = torch.randn(2 * L, R, generator=gen), (torch.randn(H * d, R, generator=gen) * 0.5).to(dtype)
    t["z"] = (torch.tanh(low).double() @ w2.double().T).float()
    want, states = _wkv_plain(t, H, d, [(0, L), (L, 2 * L)], eps)
    g = {k: v.to(DEV) for k, v in t.items()}
    state = torch.full((5, H, d, d), float("nan"), device=DEV)
    last = torch.full((5, 24), float("nan"), dtype=dtype, device=DEV)
    state[[4, 1]] = 0.0
    tok_slot = torch.tensor(slots, dtype=torch.int32, device=DEV)
    outs = []
    for i in range(L):
        rows = [i, i, L + i]
        p = torch.cat([g[k][rows].float() for k in "rkvg"] + [low[rows].to(DEV)], dim=1)      # column ranges of one row, as the products leave them
        r, k, v, gt, lw = p.split([H * d] * 4 + [R], dim=1)
        out = torch.empty((3, H * d), dtype=dtype, device=DEV)
        K().wkv_decode(r, k, v, gt, lw, w2.to(DEV), g["w0"], g["u"], g["norm"], eps, g["h"][rows].contiguous(), last, tok_slot, state, out)
        outs.append(out[[0, 2]])
    got = torch.stack(outs, 1).reshape(2 * L, H * d)
    assert rel(got, want) <= (3e-5 if dtype == torch.float32 else 6e-3)
    for s, S in zip((4, 1), states):
        assert rel(state[s], S) <= 2e-5
    assert torch.equal(last[4], g["h"][L - 1]) and torch.equal(last[1], g["h"][2 * L - 1]) and torch.isnan(state[[0, 2, 3]]).all()


@pytest.mark.parametrize("m", [1, 3, 8, 13])
@pytest.mark.parametrize("k, rows, rest", [(256, 48, 16), (256, 16, 5), (512, 64, 1), (1024, 2048, 64)])
def test_products_of_several_mixtures_in_one_launch(m, k, rows, rest):
    g = torch.Generator().manual_seed(k + rest)
    a = torch.randn(5, m, k, generator=g).to(torch.bfloat16).to(DEV)
    w = (torch.randn(4 * rows + rest, k, generator=g) / math.sqrt(k)).to(torch.bfloat16).to(DEV)
    assert K().gemm_decode_groups_supported(m, k, rows)
    out = torch.full((m, 4 * rows + rest), float("nan"), device=DEV)
    K().gemm_decode_groups(a, w, out, rows)
    want = torch.cat([a[j].double() @ w[j * rows:(j + 1) * rows if j < 4 else None].double().T for j in range(5)], dim=1)
    assert float((out.double() - want).abs().max()) < 1e-4


# ----------------------------------------------------------------------------- the norm on a sublayer's output
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width, n_terms, top", [(48, 2, 0), (37, 1, 3), (1024, 0, 4), (64, 3, 2), (2044, 2, 5), (2052, 1, 0), (5000, 1, 2)])
def test_the_norm_behind_a_sublayer_and_the_one_in_front_of_the_next(dtype, width, n_terms, top):
    g = torch.Generator().manual_seed(width)
    n, eps, eps2 = 9, 1e-4, 3e-3
    x = torch.randn(n, width, generator=g)
    terms = [(torch.randn(n, width, generator=g).to(dtype), 0.5 + i) for i in range(n_terms)]
    rows = torch.randn(n * top, width, generator=g).to(dtype) if top else None
    wts = torch.rand(n, top, generator=g) if top else None
    f, w = 1.0 + 0.3 * torch.randn(width, generator=g), 1.0 + 0.3 * torch.randn(width, generator=g)
    y = sum((t.double() * s for t, s in terms), torch.zeros(n, width, dtype=F))
    if top:
        y = y + (rows.double().view(n, top, width) * wts.double()[:, :, None]).sum(1)
    want = x.double() + P.unit_rms(y, eps) * f.double()
    want_h = P.unit_rms(want, eps2) * w.double()
    for with_norm in (True, False):
        xs, h = x.to(DEV), torch.empty((n, width), dtype=dtype, device=DEV)
        K().stream_norm_join(xs, [(t.to(DEV), s) for t, s in terms], factor=f.to(DEV), eps=eps, rows=rows.to(DEV) if top else None,
                             wts=wts.to(DEV) if top else None, norm_w=w.to(DEV) if with_norm else None, norm_eps=eps2, h=h if with_norm else None)
        assert rel(xs, want) <= 1e-6
        if with_norm:
            assert rel(h, want_h) <= (2e-6 if dtype == torch.float32 else 5e-3)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n, F_, ld", [(3, 64, 64), (5, 37, 40), (9, 2056, 2064)])
def test_the_square_of_relu(dtype, n, F_, ld):
    z = torch.randn(n, ld, generator=torch.Generator().manual_seed(F_)).to(dtype).to(DEV)
    out = torch.empty((n, F_), dtype=dtype, device=DEV)
    K().relu2(z[:, :F_], out)
    assert rel(out, torch.clamp(z[:, :F_].double().cpu(), min=0.0) ** 2) <= (1e-6 if dtype == torch.float32 else 5e-3)
