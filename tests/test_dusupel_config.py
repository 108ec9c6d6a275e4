"""The Dusupel configuration on the CPU: keys and the errors that name them, the spec and the tensors it expects against the
tests' own weights, ranks that only the tensors carry, the run order, accounting, pages of kept first tokens; and properties of
the plain mechanisms the GPU tests compare with: the delta rule against its closed forms, the window's and the kept tokens'
edges, the convolution's column order, the rotation's pairs, the layer norm."""

import copy
import json
import math
import os

import pytest
import torch

import dusupel_models as M
import plain_dusupel as P
from dryft_b200.cache import KVNeed, PageLedger, SequenceCache, StateNeed
from dryft_b200.config import ConfigError, DusupelConfig, config_from_dict, load_config, preset
from dryft_b200.config.presets import EQUAL_SIZE
from dryft_b200.weights import Checkpoint, expected_tensors, write_random_model
from dryft_b200.weights.checkpoint import WeightsError


# ----------------------------------------------------------------------------- configuration and tensors
@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_expected_tensors_are_the_tests_own_weights(tmp_path, name):
    cfg = M.CONFIGS[name]
    typed = config_from_dict(cfg)
    assert isinstance(typed, DusupelConfig) and DusupelConfig.from_dict(typed.to_dict()) == typed
    d = M.write_model(cfg, M.draw_weights(cfg, 1), str(tmp_path))
    spec = load_config(d).model_spec()
    Checkpoint(d).check(expected_tensors(spec))      # every name, every shape; the low ranks are the tensors' own
    assert [s.layer for s in spec.schedule] == P.run_order(cfg) == typed.run_order()
    assert all(s.enter is None and s.cache_from is None for s in spec.schedule)


def test_a_rank_is_free_but_nothing_else_is(tmp_path):
    cfg = M.CONFIGS["delta"]
    w = M.draw_weights(cfg, 1)
    for name, shape, ok in (("l0.mix.a1", (9, 48), True), ("l0.mix.a1", (9, 47), False), ("l0.mix.q", (25, 48), False), ("l0.mix.g2", (80, 4), True),
                            ("l0.mix.g2", (81, 5), False), ("l0.mix.a1", (9,), False)):
        d = M.write_model(cfg, dict(w, **{name: torch.zeros(shape, dtype=torch.bfloat16)}), str(tmp_path / f"{name}{shape}"))
        check = lambda: Checkpoint(d).check(expected_tensors(load_config(d).model_spec()))
        if ok:
            check()
        else:
            with pytest.raises(WeightsError, match=name.replace(".", r"\.")):
                check()


def test_a_layer_without_a_feed_forward_may_hold_its_norm(tmp_path):
    cfg = M.config([M.delta(ff=None)])
    w = M.draw_weights(cfg, 1)
    for i, more in enumerate(({}, {"l0.norm2": torch.ones(48), "l0.norm2.b": torch.zeros(48)})):
        d = M.write_model(cfg, dict(w, **more), str(tmp_path / str(i)))
        Checkpoint(d).check(expected_tensors(load_config(d).model_spec()))
    d = M.write_model(cfg, dict(w, **{"l0.norm3": torch.ones(48)}), str(tmp_path / "x"))
    with pytest.raises(WeightsError, match="norm3"):
        Checkpoint(d).check(expected_tensors(load_config(d).model_spec()))


def test_errors_name_the_key():
    base = M.CONFIGS["looped"]

    def broken(change):
        raw = copy.deepcopy(base)
        change(raw)
        return raw

    cases = [
        (lambda r: r.pop("vocab"), "vocab"), (lambda r: r.update(width=0), "width"), (lambda r: r["norm"].update(eps=-1.0), "norm.eps"),
        (lambda r: r.update(residual_mult="a"), "residual_mult"), (lambda r: r.update(layers=[]), "layers"),
        (lambda r: r["layers"][0].update(type="attention"), "layers\\[0\\].type"), (lambda r: r["layers"][0]["mixer"].pop("conv"), "mixer.conv"),
        (lambda r: r["layers"][0]["mixer"].update(heads=3), "multiple of kv_heads"), (lambda r: r["layers"][1]["mixer"].pop("right"), "right"),
        (lambda r: r["layers"][1]["mixer"]["left"]["rot"].update(dims=7), "rot.dims"), (lambda r: r["layers"][1]["mixer"]["left"].pop("scale"), "left.scale"),
        (lambda r: r["layers"][1]["mixer"]["left"]["mask"].update(size=0), "mask.size"),
        (lambda r: r["layers"][1]["mixer"]["left"]["mask"].update(keep_first=-1), "keep_first"),
        (lambda r: r["layers"][1]["mixer"]["left"]["rot"].update(scaling={"factor": 2.0}), "scaling"),
        (lambda r: r["layers"][0]["mlp"].update(kind="moe"), "mlp.kind"), (lambda r: r["layers"][0]["mlp"].pop("ff"), "mlp.ff"),
        (lambda r: r["loop"].update(stop=9), "loop"), (lambda r: r["loop"].update(times=0), "times"), (lambda r: r["loop"].update(start=True), "loop.start"),
    ]
    for change, key in cases:
        with pytest.raises(ConfigError, match=key):
            config_from_dict(broken(change))


def test_absent_keys():
    raw = copy.deepcopy(M.CONFIGS["pair"])
    raw.pop("residual_mult")
    m = raw["layers"][0]["mixer"]
    for key in ("left_scale", "right_scale"):
        m.pop(key)
    m["left"].pop("rot")
    m["left"].pop("mask")
    spec = config_from_dict(raw).model_spec()
    mix = spec.layers[0].mixer
    assert mix["left_scale"] == mix["right_scale"] == 1.0
    assert mix["left"]["window"] is None and mix["left"]["keep_first"] == 0 and mix["left"]["position"] is None
    assert [e.spec["mult"] for e in spec.layers[0].extra] == [1.0] and len(spec.schedule) == 1


def test_presets_and_accounting(tmp_path):
    for name in ("dusupel-tiny", "dusupel-1k", "dusupel-2k"):
        cfg = config_from_dict(preset(name))
        exp = expected_tensors(cfg.model_spec())
        per_layer = [sum(math.prod(i.shape) for n, i in exp.items() if n.startswith(f"l{k}.") and i.kind == "matrix") for k in range(cfg.num_layers)]
        total = sum(per_layer[i] for i in cfg.run_order())
        assert cfg.matmul_flops_per_token() == 2 * total
        assert cfg.weight_bytes_per_decode_step(2, 8) == 2 * (total + cfg.vocab * cfg.width)
    for name in ("dusupel-1k", "dusupel-2k"):
        a, b = config_from_dict(preset(name)), config_from_dict(preset(EQUAL_SIZE[name]))
        assert (a.width, a.vocab, len(a.run_order())) == (b.width, b.vocab, len(b.run_order()))
    d = write_random_model(preset("dusupel-tiny"), 3, str(tmp_path / "m"))
    assert json.load(open(os.path.join(d, "config.json")))["architecture"] == "Dusupel"
    Checkpoint(d).check(expected_tensors(load_config(d).model_spec()))


# ----------------------------------------------------------------------------- the cache: kept first tokens, states of a repeated layer
def test_pages_of_kept_first_tokens_stay():
    led = PageLedger(n_pages=12, page_size=16, max_pages_per_slot=20, window=40, keep_first=17)
    led.open(0)
    cur = 0
    for new in (10, 90, 91, 150, 230):
        led.grow(0, cur, new)
        led.trim(0, new)
        first = max(0, new - 40 + 1) // 16
        assert sorted(led.held(0)) == [p for p in range((new + 15) // 16) if p < 2 or p >= first]
        led.check()
        cur = new
    led.close(0)
    led.check()
    assert led.pool.n_free == 12


def test_groups_differ_by_what_they_keep():
    needs = [(KVNeed(1, 8, 32, 8, None, True, None, 0), None), (KVNeed(1, 8, 32, 8, None, True, None, 5), {"conv": StateNeed((4, 6), torch.bfloat16)})]
    cache = SequenceCache(needs, [None, None], max_tokens=512, max_slots=2, max_seq_len=256, page_size=16, dtype=torch.float32, device=torch.device("cpu"))
    s, = cache.open_sequences(1)
    for _ in range(6):
        cache.reserve(s, 30)
        cache.advanced(s, 30)
    assert sorted(cache._groups[0].ledger.held(s)) == [9, 10, 11] and sorted(cache._groups[1].ledger.held(s)) == [0, 9, 10, 11]
    assert cache.state(1)["conv"].dtype == torch.bfloat16
    cache.close_sequences([s])
    cache.check()


# ----------------------------------------------------------------------------- properties of the plain mechanisms
def test_the_delta_rule_overwrites_what_a_key_held():
    """Without decay, with beta = 1 and orthogonal unit keys: writing a key again replaces its value, others stay."""
    e = torch.eye(4, dtype=torch.float64)
    k = torch.stack([e[0], e[1], e[0], e[2]])[:, None]
    v = torch.tensor([[1.0, 2.0], [3.0, 4.0], [5.0, 6.0], [7.0, 8.0]], dtype=torch.float64)[:, None]
    o, S = P.delta_rule(k, k, v, torch.zeros(4, 1, 1, dtype=torch.float64), torch.ones(4, 1, dtype=torch.float64))
    assert torch.equal(o, v)                                  # the read-out sees the token's own write
    assert torch.equal(S[0], torch.stack([v[2, 0], v[1, 0], v[3, 0], torch.zeros(2, dtype=torch.float64)]))


def test_the_delta_rule_decays_before_it_corrects():
    """Two writes along one key: S2 = g S1 + k beta (v2 - g S1^T k); a decay per channel acts on the rows of the state."""
    torch.manual_seed(0)
    k = P.unit(torch.randn(1, 1, 3, dtype=torch.float64)).repeat(2, 1, 1)
    v, lg, beta = torch.randn(2, 1, 2).double(), -torch.rand(2, 1, 3).double(), torch.rand(2, 1).double()
    o, S = P.delta_rule(k, k, v, lg, beta)
    S1 = torch.outer(k[0, 0], beta[0, 0] * v[0, 0])
    D = torch.exp(lg[1, 0])[:, None] * S1
    S2 = D + torch.outer(k[1, 0], beta[1, 0] * (v[1, 0] - D.T @ k[1, 0]))
    assert torch.allclose(S[0], S2, atol=1e-14) and torch.allclose(o[1, 0], S2.T @ k[1, 0], atol=1e-14)


def test_a_decay_per_head_is_a_decay_per_channel_that_is_the_same_everywhere():
    torch.manual_seed(1)
    q, k, v = torch.randn(9, 2, 5).double(), torch.randn(9, 2, 5).double(), torch.randn(9, 2, 3).double()
    lg, beta = -torch.rand(9, 2, 1).double(), torch.rand(9, 2).double()
    a, b = P.delta_rule(q, k, v, lg, beta), P.delta_rule(q, k, v, lg.expand(9, 2, 5), beta)
    assert torch.allclose(a[0], b[0]) and torch.allclose(a[1], b[1])


def test_the_rule_is_the_same_in_pieces():
    torch.manual_seed(2)
    args = [torch.randn(11, 2, 4).double(), P.unit(torch.randn(11, 2, 4).double()), torch.randn(11, 2, 3).double(), -torch.rand(11, 2, 4).double(), torch.rand(11, 2).double()]
    o, S = P.delta_rule(*args)
    o1, S1 = P.delta_rule(*(t[:5] for t in args))
    o2, S2 = P.delta_rule(*(t[5:] for t in args), S=S1)
    assert torch.allclose(torch.cat([o1, o2]), o) and torch.allclose(S2, S)


@pytest.mark.parametrize("size, keep", [(1, 0), (5, 2), (4, 9), (30, 3)])
def test_what_a_position_sees(size, keep):
    mask = {"size": size, "keep_first": keep}
    vis = P.visible(20, mask)
    for i in range(20):
        seen = {j for j in range(20) if vis[i, j]}
        assert seen == {j for j in range(20) if P.sees(i, j, mask)} == ({*range(max(0, i - size + 1), i + 1)} | {j for j in range(keep) if j <= i})
    assert torch.equal(P.visible(6, None), torch.ones(6, 6, dtype=torch.bool).tril())


def test_convolution_rotation_and_norm():
    u, w = torch.arange(1.0, 7.0).double()[:, None], torch.tensor([[100.0, 10.0, 1.0]]).double()
    assert P.short_conv(u, w)[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0, 345.0, 456.0]       # the last column is the current token's
    v = torch.zeros(1, 1, 6, dtype=torch.float64)
    v[0, 0, 0], v[0, 0, 5] = 1.0, 3.0
    r = P.rotate_halves(v, torch.tensor([2]), {"dims": 4, "base": 100.0})[0, 0]              # dims 0 and 2 turn together; dim 5 stays
    assert torch.allclose(r, torch.tensor([math.cos(2.0), 0.0, math.sin(2.0), 0.0, 0.0, 3.0], dtype=torch.float64))
    r = P.rotate_halves(torch.eye(4, dtype=torch.float64)[1].view(1, 1, 4), torch.tensor([3]), {"dims": 4, "base": 100.0})[0, 0]
    assert torch.allclose(r, torch.tensor([0.0, math.cos(0.3), 0.0, math.sin(0.3)], dtype=torch.float64))
    x = torch.tensor([[1.0, 3.0]], dtype=torch.float64)
    assert torch.allclose(P.layer_norm(x, torch.tensor([2.0, 2.0]).double(), torch.tensor([0.5, 0.5]).double(), 0.0), torch.tensor([[-1.5, 2.5]]).double())
