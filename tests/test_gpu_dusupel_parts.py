"""The kernels of the Dusupel design alone against the plain functions (``plain_dusupel.py``): the gated delta rule over prompts
and token by token, with a write hundreds of tokens back that still decides an output, at sizes that fit no vector, no warp and
no group of four tokens; the attention that keeps the first tokens, with ONE key that outweighs all others placed at every
edge of the window, of the kept tokens and of a page; short convolutions across the cuts of a prompt; the rotation behind them;
the gate per value; two layer norms in the launch that forms the stream's sum."""

import types

import numpy as np
import pytest
import torch

import plain_dusupel as P

pytestmark = pytest.mark.gpu
DEV = "cuda"


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def step_context(lens, starts, slots, tile=64):
    """What a step of these pieces looks like to the kernels (tiles listed in no particular order)."""
    cu = [0] + list(np.cumsum(lens))
    t0, tn = [], []
    for b, n in enumerate(lens):
        for a in range(0, n, tile):
            t0.append(cu[b] + a)
            tn.append(min(tile, n - a))
    order = sorted(range(len(t0)), key=lambda i: -t0[i] % 7)
    return types.SimpleNamespace(
        tile_tok0=i32([t0[i] for i in order]), tile_rows=i32([tn[i] for i in order]), n_tiles=len(t0), tile_size=tile, cu_q=i32(cu), n_seqs=len(lens),
        seq_slot=i32(slots), tok_slot=i32([s for s, n in zip(slots, lens) for _ in range(n)]),
        tok_pos=i32([st + i for st, n in zip(starts, lens) for i in range(n)]))


def plain_rule(x, dec, logit, cw, a_log, dt_bias, H, G, d, dv, per_channel):
    """The plain functions over one whole sequence of projected rows ``x [L, 2 G d + H dv]``."""
    L = x.shape[0]
    y = P.silu(P.short_conv(x, cw))
    q, k = P.unit(y[:, :G * d].view(L, G, d)) * d ** -0.5, P.unit(y[:, G * d:2 * G * d].view(L, G, d))
    q, k = (t.repeat_interleave(H // G, dim=1) for t in (q, k))
    z = P.softplus(dec + dt_bias)
    lg = -torch.exp(a_log)[:, None] * (z.view(L, H, d) if per_channel else z[..., None])
    return P.delta_rule(q, k, y[:, 2 * G * d:].view(L, H, dv), lg, torch.sigmoid(logit))


SIZES = [(1, 1, 16, 16, 4), (4, 2, 10, 18, 3), (3, 3, 1, 3, 5), (2, 1, 33, 40, 1), (6, 2, 64, 7, 2), (2, 2, 100, 33, 4), (4, 4, 128, 128, 4),
         (1, 1, 200, 20, 6)]


@pytest.mark.parametrize("per_channel", [False, True])
@pytest.mark.parametrize("H, G, d, dv, taps", SIZES)
def test_gated_delta_rule_remembers_hundreds_of_tokens(H, G, d, dv, taps, per_channel):
    """Several unequal sequences in one step (one of a single token, one of two), the first cut at an odd place, then a few
    single tokens.  Head 0 of the first sequence writes strongly once, near its start, forgets next to nothing and writes next to
    nothing else: its outputs 600 tokens later still read that one write."""
    from dryft_b200.ops import kernels as K

    torch.manual_seed(100 * d + dv)
    lens, slots, tail = [650, 1, 37, 2, 130], [4, 0, 2, 6, 1], 6
    CH = 2 * G * d + H * dv
    full = [n + tail for n in lens]
    ld, x_off, b_off = CH + 2 * H + 5, 3, CH + 4
    n_dec = H * d if per_channel else H
    seqs = []
    for b, n in enumerate(full):
        x = torch.randn(n, CH)
        logit = torch.randn(n, H) * 2.0
        dec = torch.randn(n, n_dec) - 1.0
        if b == 0:
            logit[:, 0] = -14.0
            logit[20, 0] = 9.0
            x[20, 2 * G * d:2 * G * d + dv] = 12.0
            dec[:, :n_dec // H] = -14.0
        seqs.append((x, logit, dec))
    cw = torch.randn(CH, taps) * 0.4
    cw[:, -1] += 0.8
    a_log, dt_bias, norm_w = torch.randn(H) * 0.5, torch.randn(n_dec) * 0.3, 1.0 + 0.3 * torch.randn(dv)
    f = lambda t: t.double()
    want = [plain_rule(f(x), f(dec), f(lg), f(cw), f(a_log), f(dt_bias), H, G, d, dv, per_channel)[0] for x, lg, dec in seqs]
    gates = [torch.randn(n, H * dv) for n in full]
    eps = 1e-5
    outs = [P.gated_head_norm(o, f(norm_w), P.silu(f(g)), eps) for o, g in zip(want, gates)]
    # the one write is what head 0 reads at the end: without it the outputs of the last tokens are next to nothing
    x, lg, dc = (f(t).clone() for t in seqs[0])
    lg[20, 0] = -14.0
    without = plain_rule(x, dc, lg, f(cw), f(a_log), f(dt_bias), H, G, d, dv, per_channel)[0]
    assert float(want[0][-40:, 0].abs().max()) > 100.0 * float(without[-40:, 0].abs().max())

    state = torch.full((8, H, dv, K.delta_state_rows(d)), float("nan"), device=DEV)
    ring = torch.full((8, taps, CH), float("nan"), device=DEV) if taps > 1 else None
    for s in slots:
        state[s] = 0.0
    c = lambda t: t.to(DEV).contiguous()
    consts = (c(cw), ring, c(a_log), c(dt_bias), c(norm_w), eps, False)

    def rows(pieces):
        proj = torch.zeros(sum(e - a for _, a, e in pieces), ld)
        at, dec, gate = 0, [], []
        for b, a, e in pieces:
            x, logit, dc = seqs[b]
            proj[at:at + e - a, x_off:x_off + CH] = x[a:e]
            proj[at:at + e - a, b_off:b_off + H] = logit[a:e]
            dec.append(dc[a:e])
            gate.append(gates[b][a:e])
            at += e - a
        return c(proj), c(torch.cat(dec)), c(torch.cat(gate))

    def compare(out, pieces, what):
        at = 0
        for b, a, e in pieces:
            err = (out[at:at + e - a].double().cpu() - outs[b][a:e]).abs().amax(dim=1)
            # the norm divides by the output's own size: a row whose output all but vanishes magnifies the rounding of what the
            # state holds (the one strong write is there in every row)
            size = want[b].abs().max()
            small = torch.sqrt((want[b][a:e] ** 2).mean(-1)).amin(dim=1) + eps ** 0.5
            tol = 3e-5 * outs[b][a:e].abs().max() + 1e-5 * size / small
            assert bool((err <= tol).all()), f"{what}: sequence {b}, token {a + int((err - tol).argmax())} off by {float(err.max()):.3g}"
            at += e - a

    # the first 333 tokens of sequence 0 and all of the others, then the rest of sequence 0, then single tokens
    cut = 333
    for pieces in ([(0, 0, cut)] + [(b, 0, lens[b]) for b in range(1, len(lens))], [(0, cut, lens[0])]):
        ctx = step_context([e - a for _, a, e in pieces], [a for _, a, _ in pieces], [slots[b] for b, _, _ in pieces])
        proj, dec, gate = rows(pieces)
        out = torch.full((proj.shape[0], H * dv), float("nan"), device=DEV)
        K.delta_tokens(proj, x_off, b_off, dec, gate, *consts, ctx, state, out, H, G, d, dv, per_channel)
        compare(out, pieces, "many tokens")
    for t in range(tail):
        pieces = [(b, lens[b] + t, lens[b] + t + 1) for b in range(len(lens))]
        proj, dec, gate = rows(pieces)
        # a padding row at the end: nothing of it is read, and its output is zeros
        proj, dec, gate = (torch.cat([m, torch.full_like(m[:1], float("nan"))]) for m in (proj, dec, gate))
        out = torch.full((len(pieces) + 1, H * dv), float("nan"), device=DEV)
        K.delta_decode(proj, x_off, b_off, dec, gate, *consts, i32(slots + [-1]), i32([lens[b] + t for b in range(len(lens))] + [0]), state, out, H,
                       G, d, dv, per_channel)
        compare(out[:-1], pieces, "single tokens")
        assert float(out[-1].abs().max()) == 0.0
    # the state itself, transposed, with zeros behind the key size
    for b, s in enumerate(slots):
        x, lg, dc = seqs[b]
        S = plain_rule(f(x), f(dc), f(lg), f(cw), f(a_log), f(dt_bias), H, G, d, dv, per_channel)[1]
        got = state[s].double().cpu()
        assert float((got[..., :d].transpose(1, 2) - S).abs().max()) <= 2e-5 * max(1.0, float(S.abs().max())), f"state of sequence {b}"
        assert float(got[..., d:].abs().sum()) == 0.0
    untouched = [s for s in range(8) if s not in slots]
    assert torch.isnan(state[untouched]).all()
    if taps > 1:
        assert torch.isnan(ring[untouched]).all()


@pytest.mark.parametrize("H, G, d, dv, taps", [(4, 2, 128, 128, 4), (2, 2, 64, 32, 4)])
def test_gated_delta_rule_reads_bfloat16_rows(H, G, d, dv, taps):
    """Rows in bfloat16 (and a column slice as gate): the same as the 32-bit kernels over the same values, up to the rounding
    of the result; the walk gives a sequence the same bits alone and beside others."""
    from dryft_b200.ops import kernels as K

    torch.manual_seed(d)
    lens, CH = [200, 70], 2 * G * d + H * dv
    n, ld = sum(lens), (CH + H + H * dv + 7) // 8 * 8
    proj = torch.randn(n, ld, device=DEV).to(torch.bfloat16)
    dec = (torch.randn(n, H * d, device=DEV) - 1.0).to(torch.bfloat16)
    cw, a_log, dtb, nw = torch.randn(CH, taps, device=DEV) * 0.5, torch.randn(H, device=DEV), torch.randn(H * d, device=DEV), torch.ones(dv, device=DEV)

    def run(p, dc, ln, dtype):
        st = torch.zeros(2, H, dv, K.delta_state_rows(d), device=DEV)
        ring = torch.zeros(2, taps, CH, device=DEV, dtype=dtype)
        out = torch.empty(p.shape[0], H * dv, device=DEV, dtype=dtype)
        K.delta_tokens(p, 0, CH, dc, p[:, CH + H:CH + H + H * dv], cw, ring, a_log, dtb, nw, 1e-5, True, step_context(ln, [0] * len(ln), list(range(len(ln)))),
                       st, out, H, G, d, dv, True)
        return out, st, ring

    out, st, ring = run(proj, dec, lens, torch.bfloat16)
    ref, st32, _ = run(proj.float(), dec.float(), lens, torch.float32)
    assert torch.equal(st, st32)
    assert float((out.float() - ref).abs().max()) <= 2 ** -8 * float(ref.abs().max())
    alone, st1, ring1 = run(proj[:lens[0]].contiguous(), dec[:lens[0]].contiguous(), lens[:1], torch.bfloat16)
    assert torch.equal(alone, out[:lens[0]]) and torch.equal(st1[0], st[0]) and torch.equal(ring1[0], ring[0])


# ----------------------------------------------------------------------------- attention that keeps the first tokens
@pytest.mark.parametrize("size, keep", [(50, 3), (64, 64), (129, 70), (1, 5), (3, 0), (200, 130)])
@pytest.mark.parametrize("edge", ["first", "last kept", "first not kept", "page", "late"])
def test_one_key_that_stands_out_at_every_edge(size, keep, edge):
    """Both attention kernels (row-wise in 32-bit with several splits, prompts in bfloat16) against the plain function over 500
    tokens in which ONE key outweighs all others for every query: seen for ever if it is among the first ``keep``, else until the
    window has passed it.  Pages that hold neither kept tokens nor any of a query's window are NaN."""
    from dryft_b200.ops import kernels as K

    torch.manual_seed(size + keep)
    page, n_kv, group, d, dv, L = 64, 2, 2, 16, 32, 500
    far = {"first": 0, "last kept": max(keep - 1, 0), "first not kept": keep, "page": 63, "late": 320}[edge]
    H = n_kv * group
    k = (0.1 * torch.randn(L, n_kv, d)).to(torch.bfloat16).double()
    v = torch.randn(L, n_kv, dv).to(torch.bfloat16).double()
    q = torch.zeros(L, H, d, dtype=torch.float64)
    q[:, :, 3] = 1.0
    k[far, :, 3] = 40.0
    v[far] = 7.0
    gate = torch.randn(L, H * dv).to(torch.bfloat16).double()
    seen = P.visible(L, {"size": size, "keep_first": keep})
    plain = torch.stack([P.masked_softmax_attention(q[:, h], k[:, h // group], v[:, h // group], 1.5, seen) for h in range(H)], dim=1)
    want = plain * torch.sigmoid(gate).view(L, H, dv)
    out_at = far + size      # the first position whose window has passed the key
    assert float(plain[min(out_at - 1, L - 1), 0, 0]) > 6.0
    if out_at < L:
        assert (float(plain[out_at, 0, 0]) > 6.0) == (far < keep)
    n_pages = 9
    table = torch.randperm(n_pages)[None].to(torch.int32).to(DEV)
    k32 = torch.full((n_pages, n_kv, page, d), float("nan"), device=DEV)
    v32 = torch.full((n_pages, n_kv, page, dv), float("nan"), device=DEV)
    for j in range(L):
        k32[table[0, j // page], :, j % page] = k[j].float().to(DEV)
        v32[table[0, j // page], :, j % page] = v[j].float().to(DEV)
    g32 = torch.cat([torch.zeros(L, 3), gate.float()], dim=1).to(DEV)[:, 3:]        # a column slice
    for first in (0, 257, 449):      # all positions; later ones over pages of which only the ones in sight are left
        kk, vv = k32.clone(), v32.clone()
        for pg in range(n_pages):
            if pg * page >= keep and (pg + 1) * page <= first - size + 1:
                kk[table[0, pg]], vv[table[0, pg]] = float("nan"), float("nan")
        n = L - first
        tok_slot, tok_pos = i32([0] * n), i32(list(range(first, L)))
        qq = q[first:].float().to(DEV)
        got = torch.empty(n, H, dv, device=DEV)
        for splits in (1, 3, 5):
            po = torch.empty(n, H, splits, dv, device=DEV) if splits > 1 else None
            pm = torch.empty(n, H, splits, 2, device=DEV) if splits > 1 else None
            K.pool_attn_rows(qq, kk, vv, table, None, None, tok_slot, tok_pos, got, 1.5, size, 0, splits, po, pm, keep=keep, gate=g32[first:])
            err = (got.double().cpu() - want[first:]).abs().amax(dim=(1, 2))
            assert float(err.max()) <= 2e-5, f"{splits} split(s), from {first}: position {first + int(err.argmax())} off by {float(err.max()):.3g}"
        bf = lambda x: x.to(torch.bfloat16).contiguous()
        t0 = list(range(0, n, 64))
        gotb = torch.empty(n, H, dv, device=DEV, dtype=torch.bfloat16)
        for cols in (bf(g32[first:]), bf(torch.cat([torch.zeros(n, 3, device=DEV), g32[first:]], dim=1))[:, 3:]):     # aligned and odd columns
            K.pool_attn_prefill(bf(qq), bf(kk), bf(vv), table, None, None, i32(t0), i32([min(64, n - a) for a in t0]), tok_slot, tok_pos, gotb,
                                len(t0), 1.5, size, 0, keep=keep, gate=cols)
            errb = (gotb.double().cpu() - want[first:]).abs().amax(dim=(1, 2))
            assert float(errb.max()) <= 0.06, f"prompt kernel from {first}: position {first + int(errb.argmax())} off by {float(errb.max()):.3g}"


@pytest.mark.parametrize("taps", [1, 2, 4, 7])
@pytest.mark.parametrize("rot", [0, 6, 16])
@pytest.mark.parametrize("runs", [False, True])      # token by token, or runs of tokens where the step has many
def test_convolved_rotated_queries_keys_and_values_across_cuts(taps, rot, runs):
    """The preparation of a head behind a short convolution: whole prompts, pieces shorter than the taps, single tokens; two
    sequences in a step, their slots' rings NaN before (what is not of the sequence is never read)."""
    from dryft_b200.ops import kernels as K

    torch.manual_seed(10 * taps + rot)
    H, G, d, dv, page = 4, 2, 16, 12, 64
    CH, L = H * d + G * (d + dv), 90
    cw = torch.randn(CH, taps)
    xs = [torch.randn(L, CH) for _ in range(2)]
    freq = torch.pow(torch.tensor(50.0, dtype=torch.float64), -2.0 * torch.arange(rot // 2, dtype=torch.float64) / rot) if rot else None
    lo = (freq - freq.float().double()).float().to(DEV) if rot else None
    pos = torch.arange(L)
    rt = {"dims": rot, "base": 50.0} if rot else None
    want = []
    for x in xs:
        y = P.short_conv(x.double(), cw.double())
        want.append((P.rotate_halves(y[:, :H * d].view(L, H, d), pos, rt), P.rotate_halves(y[:, H * d:(H + G) * d].view(L, G, d), pos, rt),
                     y[:, (H + G) * d:].view(L, G, dv)))
    table = i32([[0, 1], [2, 3], [4, 5]])
    kp, vp = torch.zeros(6, G, page, d, device=DEV), torch.zeros(6, G, page, dv, device=DEV)
    ring = torch.full((3, taps, CH), float("nan"), device=DEV) if taps > 1 else None
    slots, cw_d = [2, 0], cw.to(DEV)
    at = [0, 0]
    for lens in ([37, 1], [2, 3], [1, 1], [1, 1], [3, 50], [1, 1], [45, 33]):
        x = torch.cat([torch.cat([xs[b][at[b]:at[b] + n], torch.zeros(n, 5)], dim=1) for b, n in enumerate(lens)]).to(DEV).contiguous()
        ctx = step_context(lens, at, slots)
        q = torch.empty(sum(lens), H, d, device=DEV)
        decode = all(n == 1 for n in lens)
        if runs and not decode:
            K.pool_attn_prep_run(x, freq.float().to(DEV) if rot else None, lo, rot, ctx, q, kp, vp, table, H, G, -1.0, cw_d, ring)
        else:
            K.pool_attn_prep(x, None, None, None, freq.float().to(DEV) if rot else None, lo, rot, ctx.tok_slot, ctx.tok_pos, q, kp, vp, table, H, G, -1.0, True,
                             conv_w=cw_d, ring=ring, store_ring=decode)
        if taps > 1 and not decode:
            K.conv_ring_store(x, 0, ctx.cu_q, ctx.seq_slot, ctx.tok_pos, ring, len(lens))
        o = 0
        for b, n in enumerate(lens):
            sl = slice(at[b], at[b] + n)
            assert float((q[o:o + n].double().cpu() - want[b][0][sl]).abs().max()) <= 1e-5, f"queries of sequence {b} from {at[b]}"
            for i in range(at[b], at[b] + n):
                pg = int(table[slots[b], i // page])
                assert float((kp[pg, :, i % page].double().cpu() - want[b][1][i]).abs().max()) <= 1e-5, f"key {i} of sequence {b}"
                assert float((vp[pg, :, i % page].double().cpu() - want[b][2][i]).abs().max()) <= 1e-5, f"value {i} of sequence {b}"
            at[b] += n
            o += n


# ----------------------------------------------------------------------------- sums and layer norms
@pytest.mark.parametrize("width", [1, 7, 256, 1000, 2048])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_sum_of_results_and_two_layer_norms(width, dtype):
    from dryft_b200.ops import kernels as K

    torch.manual_seed(width)
    n, eps = 9, 1e-5
    x = (torch.randn(n, width) + 300.0).to(DEV)            # a mean far from zero: squares of the values would lose the variance
    ys = [torch.randn(n, width).to(dtype).to(DEV) for _ in range(3)]
    w = [torch.randn(width, device=DEV) for _ in range(4)]
    scales = [0.7, -1.3, 0.25]
    for n_terms in (0, 1, 3):
        for n_norms in (0, 1, 2):
            got = x.clone()
            outs = [torch.empty(n, width, dtype=dtype, device=DEV) for _ in range(n_norms)]
            K.stream_sum_ln(got, [(y, s) for y, s in zip(ys[:n_terms], scales)], norms=[(w[2 * i], w[2 * i + 1], o) for i, o in enumerate(outs)], eps=eps)
            want = x.double() + sum(s * y.double() for y, s in zip(ys[:n_terms], scales))
            assert float((got.double() - want).abs().max()) <= 1e-4
            for i, o in enumerate(outs):
                ln = P.layer_norm(got.double().cpu(), w[2 * i].double().cpu(), w[2 * i + 1].double().cpu(), eps)
                tol = 2e-4 if dtype == torch.float32 else 2 ** -8 * float(ln.abs().max()) + 2e-4
                assert float((o.double().cpu() - ln).abs().max()) <= tol
    rows = i32([8, 0, 3])
    out = torch.empty(3, width, dtype=dtype, device=DEV)
    K.stream_sum_ln(x, norms=[(w[0], w[1], out)], eps=eps, rows=rows)
    ln = P.layer_norm(x.double().cpu()[[8, 0, 3]], w[0].double().cpu(), w[1].double().cpu(), eps)
    assert float((out.double().cpu() - ln).abs().max()) <= (2e-4 if dtype == torch.float32 else 2 ** -8 * float(ln.abs().max()) + 2e-4)
