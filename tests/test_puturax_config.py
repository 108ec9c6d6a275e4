"""The Puturax configuration on the CPU: keys and the errors that name them, the spec and the tensors it expects against the
tests' own weights, a rank that only the tensors carry, accounting; and properties of the plain mechanisms the GPU tests
compare with: the recurrence against its closed forms and in pieces, the bonus, the token before, the distance's logarithm, the
squashed score, the one in the denominator, the temperature's steps, groups and corrections, the rotation's pairs."""

import copy
import json
import math
import os

import pytest
import torch

import plain_puturax as P
import puturax_models as M
from dryft_b200.config import ConfigError, PuturaxConfig, config_from_dict, load_config, preset
from dryft_b200.config.presets import EQUAL_SIZE
from dryft_b200.weights import Checkpoint, expected_tensors, write_random_model
from dryft_b200.weights.checkpoint import WeightsError

F = torch.float64


# ----------------------------------------------------------------------------- configuration and tensors
@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_expected_tensors_are_the_tests_own_weights(tmp_path, name):
    cfg = M.CONFIGS[name]
    typed = config_from_dict(cfg)
    assert isinstance(typed, PuturaxConfig) and PuturaxConfig.from_dict(typed.to_dict()) == typed
    d = M.write_model(cfg, M.draw_weights(cfg, 1), str(tmp_path))
    spec = load_config(d).model_spec()
    Checkpoint(d).check(expected_tensors(spec))
    assert [s.layer for s in spec.schedule] == list(range(len(cfg["layers"])))


def test_a_rank_is_free_but_nothing_else_is(tmp_path):
    cfg = M.CONFIGS["pair"]
    w = M.draw_weights(cfg, 1)
    for name, shape, ok in (("l0.mix.right.w1", (9, 48), True), ("l0.mix.right.w1", (9, 47), False), ("l0.mix.right.w2", (48, 4), True),
                            ("l0.mix.right.w2", (47, 5), False), ("l0.mix.left.r1", (5,), False), ("l0.mix.right.u", (48,), False),
                            ("l0.norm1b", (47,), False)):
        d = M.write_model(cfg, dict(w, **{name: torch.zeros(shape, dtype=torch.bfloat16)}), str(tmp_path / f"{name}{shape}"))
        check = lambda: Checkpoint(d).check(expected_tensors(load_config(d).model_spec()))
        if ok:
            check()
        else:
            with pytest.raises(WeightsError, match=name.replace(".", r"\.")):
                check()


def test_a_layer_without_a_feed_forward_may_hold_its_norms(tmp_path):
    cfg = M.config([M.latent(mlp=None)])
    w = M.draw_weights(cfg, 1)
    for i, more in enumerate(({}, {"l0.norm2": torch.ones(48), "l0.norm2b": torch.zeros(48)})):
        d = M.write_model(cfg, dict(w, **more), str(tmp_path / str(i)))
        Checkpoint(d).check(expected_tensors(load_config(d).model_spec()))
    d = M.write_model(cfg, dict(w, **{"l0.norm3": torch.ones(48)}), str(tmp_path / "x"))
    with pytest.raises(WeightsError, match="norm3"):
        Checkpoint(d).check(expected_tensors(load_config(d).model_spec()))


def test_errors_name_the_key():
    base = M.CONFIGS["mixed"]

    def broken(change):
        raw = copy.deepcopy(base)
        change(raw)
        return raw

    left = lambda r: r["layers"][1]["mixer"]["left"]
    router = lambda r: r["layers"][1]["mlp"]["router"]
    cases = [
        (lambda r: r.pop("vocab"), "vocab"), (lambda r: r.update(width=0), "width"), (lambda r: r["norm"].update(eps=-1.0), "norm.eps"),
        (lambda r: r["embedding"].update(scale="a"), "embedding.scale"), (lambda r: r.update(layers=[]), "layers"),
        (lambda r: r["layers"][0].update(type="attention"), "layers\\[0\\].type"), (lambda r: r["layers"][0]["mixer"].pop("q_rank"), "mixer.q_rank"),
        (lambda r: r["layers"][0]["mixer"]["rot"].update(dims=4), "rot.dims"), (lambda r: r["layers"][1]["mixer"].pop("right"), "right"),
        (lambda r: r["layers"][1]["mixer"]["right"].pop("dim"), "right.dim"), (lambda r: left(r).update(heads=3), "multiple of kv_heads"),
        (lambda r: left(r).pop("scale"), "left.scale"), (lambda r: left(r).update(softcap=0.0), "softcap"), (lambda r: left(r)["q_temp"].update(every=0), "every"),
        (lambda r: left(r)["q_temp"].update(every=2.5), "every"), (lambda r: left(r)["q_temp"].pop("coef"), "coef"),
        (lambda r: r["layers"][1]["mixer"].update(left_scale=None), "left_scale"), (lambda r: r["layers"][0]["mlp"].update(kind="glu"), "mlp.kind"),
        (lambda r: r["layers"][0]["mlp"].pop("ff"), "mlp.ff"), (lambda r: router(r).update(top=5), "router.top"),
        (lambda r: router(r)["groups"].update(count=4), "equal groups"), (lambda r: router(r)["groups"].update(keep=4), "groups"),
        (lambda r: r["layers"][1]["mlp"]["shared"].pop("ff"), "shared.ff"), (lambda r: r["layers"][1]["mlp"].pop("expert"), "expert"),
    ]
    for change, key in cases:
        with pytest.raises(ConfigError, match=key):
            config_from_dict(broken(change))


def test_absent_keys():
    raw = copy.deepcopy(M.CONFIGS["pair"])
    raw.pop("embedding")
    m = raw["layers"][0]["mixer"]
    for key in ("left_scale", "right_scale"):
        m.pop(key)
    for key in ("softcap", "q_temp"):
        m["left"].pop(key)
    raw["layers"][0]["mlp"] = M.moe(groups=None, shared=None)
    spec = config_from_dict(raw).model_spec()
    mix, ffn = spec.layers[0].mixer, spec.layers[0].ffn
    assert spec.embedding["scale"] == mix["left_scale"] == mix["right_scale"] == 1.0
    assert mix["left"]["softcap"] is None and mix["left"]["q_temp"] is None and (ffn["groups"], ffn["keep"], ffn["shared"]) == (1, 1, None)


def test_presets_and_accounting(tmp_path):
    for name in ("puturax-tiny", "puturax-1k", "puturax-2k"):
        cfg = config_from_dict(preset(name))
        exp = expected_tensors(cfg.model_spec())
        count = lambda keep: sum(math.prod(i.shape) for n, i in exp.items() if i.kind == "matrix" and keep(n))
        total = count(lambda n: ".e" not in n and n != "head")
        experts = {n.split(".")[0]: 0 for n in exp if ".mlp.e0." in n}
        for k in experts:
            experts[k] = count(lambda n: n.startswith(f"{k}.mlp.e0."))
        routers = {f"l{i}": l.mlp["router"] for i, l in enumerate(cfg.layers) if l.mlp["kind"] == "moe"}
        assert cfg.matmul_flops_per_token() == 2 * (total + sum(routers[k]["top"] * n for k, n in experts.items()))
        assert cfg.weight_bytes_per_decode_step(2, 8) == 2 * (total + cfg.vocab * cfg.width + sum(min(routers[k]["experts"], 8 * routers[k]["top"]) * n
                                                                                              for k, n in experts.items()))
    for name in ("puturax-1k", "puturax-2k"):
        a, b = config_from_dict(preset(name)), config_from_dict(preset(EQUAL_SIZE[name]))
        assert (a.width, a.vocab, len(a.layers)) == (b.width, b.vocab, len(b.run_order()))
    d = write_random_model(preset("puturax-tiny"), 3, str(tmp_path / "m"))
    assert json.load(open(os.path.join(d, "config.json")))["architecture"] == "Puturax"
    Checkpoint(d).check(expected_tensors(load_config(d).model_spec()))


# ----------------------------------------------------------------------------- properties of the plain mechanisms
def test_the_recurrence_against_its_closed_form():
    """o_t = sum over s < t of (r_t . (the decays after s, up to t - 1) k_s) v_s, plus the bonus-weighted token itself."""
    g = torch.Generator().manual_seed(0)
    L, d, dv = 7, 3, 2
    r, k = torch.randn(L, d, generator=g, dtype=F), torch.randn(L, d, generator=g, dtype=F)
    v, w, u = torch.randn(L, dv, generator=g, dtype=F), torch.rand(L, d, generator=g, dtype=F), torch.randn(d, generator=g, dtype=F)
    got = P.decayed_outer_products(r, k, v, w, u)
    for t in range(L):
        want = (r[t] * u * k[t]).sum() * v[t]
        for s in range(t):
            want = want + (r[t] * w[s + 1:t].prod(0) * k[s]).sum() * v[s]      # a token's own decay acts on what came before it
        assert torch.allclose(got[t], want, atol=1e-12)


def test_a_state_that_never_decays_sums_and_one_that_decays_at_once_forgets():
    one, zero = torch.ones(4, 1, dtype=F), torch.zeros(4, 1, dtype=F)
    v = torch.tensor([[1.0], [2.0], [3.0], [4.0]], dtype=F)
    assert P.decayed_outer_products(one, one, v, one, torch.zeros(1, dtype=F))[:, 0].tolist() == [0.0, 1.0, 3.0, 6.0]
    assert P.decayed_outer_products(one, one, v, zero, torch.full((1,), 10.0, dtype=F))[:, 0].tolist() == [10.0, 21.0, 32.0, 43.0]


def test_the_token_before_the_first_is_zero():
    h = torch.tensor([[1.0], [2.0], [5.0]], dtype=F)
    assert P.previous(h)[:, 0].tolist() == [0.0, 1.0, 2.0]


def test_scores_squashed_biased_and_shared_with_a_one():
    assert torch.allclose(P.squash(torch.tensor([0.0, 1e-3, 1e6], dtype=F), 5.0), torch.tensor([0.0, 1e-3, 5.0], dtype=F), atol=1e-9)
    assert P.squash(torch.tensor([7.0]), None).item() == 7.0
    b = P.distance_bias(4, 2.0, 3.0)
    assert torch.allclose(b[3], 2.0 * torch.log(torch.tensor([10.0, 7.0, 4.0, 1.0], dtype=F))) and float(b[0, 3]) == 0.0
    s = torch.log(torch.tensor([[1.0, 9.0], [3.0, 4.0]], dtype=F))
    assert torch.allclose(P.weights_of(s, True), torch.tensor([[0.5, 0.0], [3 / 8, 4 / 8]], dtype=F))
    assert torch.allclose(P.weights_of(s, False), torch.tensor([[1.0, 0.0], [3 / 7, 4 / 7]], dtype=F))
    low = P.weights_of(torch.full((1, 1), -800.0, dtype=F), True)                  # a score far below the one's: nothing is left
    assert float(low) == 0.0
    assert float(P.weights_of(torch.full((1, 1), 800.0, dtype=F), True)) == 1.0


def test_the_temperature_steps_behind_every_whole_stretch():
    t = P.temperature(9, {"coef": 0.5, "every": 4})
    assert torch.allclose(t, 1.0 + 0.5 * torch.log(torch.tensor([1.0, 1, 1, 2, 2, 2, 2, 3, 3], dtype=F)))      # position 3 is the fourth token
    assert torch.equal(P.temperature(3, None), torch.ones(3, dtype=F))


def test_groups_corrections_and_weights_of_a_choice():
    z = torch.tensor([[2.0, -4.0, 1.0, 0.9, -1.0, -1.0]], dtype=F)
    w = {"router": torch.eye(6, dtype=F), "correction": torch.zeros(6, dtype=F)}
    s = torch.sigmoid(z)[0]
    # groups (0, 1) (2, 3) (4, 5): the second has the larger sum, although the first holds the best expert
    idx, wts = P.router_choice(z, {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}, w, "")
    assert idx[0].tolist() == [2, 3] and torch.allclose(wts[0], s[2:4] / s[2:4].sum())
    # a correction moves the choice, not the weights; with every choice score below zero the shut-out groups stay shut out
    w["correction"] = torch.tensor([-2.0, -2.0, -5.0, -5.0, -1.4, -1.5], dtype=F)
    idx, wts = P.router_choice(z, {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}, w, "")
    assert idx[0].tolist() == [4, 5] and torch.allclose(wts[0], torch.tensor([0.5, 0.5], dtype=F))
    idx, _ = P.router_choice(z, {"experts": 6, "top": 3}, w, "")
    assert idx[0].tolist() == [0, 4, 5]


def test_rotation_and_norms():
    r = P.rotate_half(torch.eye(6, dtype=F)[1].view(1, 1, 6), torch.tensor([3]), {"dims": 4, "base": 100.0})
    assert torch.allclose(r[0, 0], torch.tensor([0.0, math.cos(0.3), 0.0, math.sin(0.3), 0.0, 0.0], dtype=F))
    x = torch.tensor([[3.0, 4.0]], dtype=F)
    assert torch.allclose(P.layer_norm1(x, torch.tensor([1.0, -0.5], dtype=F), 0.0), torch.tensor([[6.0, 2.0]], dtype=F) / math.sqrt(12.5))
    assert torch.allclose(P.plain_norm(x, torch.tensor([1.0, -0.5], dtype=F), 0.0), torch.tensor([[3.0, -2.0]], dtype=F) / math.sqrt(12.5))
