"""Host side of Rukedra models: registry, config checks, tensor names, and the plain statement of the mechanisms against closed
forms.  No device is needed."""
import copy

import numpy as np
import pytest

import plain_rukedra as P
from test_mukutar_cpu import set_config
from tl_b200 import synth

ROT = {"base": 300.0, "dims": 6, "scaling": {"factor": 2.5, "original": 50, "fast": 9.0, "slow": 1.5}}
CFG = {"architecture": "Rukedra", "vocab": 53, "width": 30, "norm": {"eps": 1e-5, "groups": 5}, "logit_softcap": 7.0, "layers": [
    {"type": "latent_attention", "mixer": {"heads": 3, "dim": 7, "rot_dim": 6, "vdim": 9, "kv_rank": 11, "q_rank": 13, "scale": 0.3, "mask": {"size": 8}, "rot": ROT},
     "mlp": {"kind": "moe", "expert": {"ff": 10}, "router": {"experts": 6, "top": 2, "scale": 1.1, "groups": {"count": 3, "keep": 2}}, "shared": {"ff": 14}}},
    {"type": "mingru", "mixer": {"width": 17}, "mlp": None},
    {"type": "latent_attention_2", "mixer": {"heads": 2, "dim": 5, "rot_dim": 6, "vdim": 4, "kv_rank": 8, "scale": 0.4, "rot": dict(ROT, scaling=None)}, "mlp": {"kind": "dense", "ff": 21}},
    {"type": "mingru", "mixer": {"width": 17}, "mlp": None, "weights_of": 1}]}


def test_registry_reads_a_config():
    st, arch, sizes = set_config(CFG)
    assert st == 0 and arch == b"Rukedra" and sizes == (4, 30, 53)


def at(*path):
    def get(c):
        for p in path:
            c = c[p]
        return c
    return get


L0, MIX, MLP = at("layers", 0), at("layers", 0, "mixer"), at("layers", 0, "mlp")


@pytest.mark.parametrize("change,status", [
    (lambda c: c.pop("width"), 8), (lambda c: c["norm"].pop("groups"), 8), (lambda c: c["norm"].update(groups=4), 8), (lambda c: c.update(logit_softcap=-1.0), 8),
    (lambda c: L0(c).update(type="attention"), 7), (lambda c: MIX(c).pop("q_rank"), 8), (lambda c: MIX(c).pop("mask"), 8), (lambda c: MIX(c).update(kv_rank=0), 8),
    (lambda c: MIX(c).pop("scale"), 8), (lambda c: MIX(c).pop("rot"), 8), (lambda c: MIX(c).update(rot_dim=4), 8), (lambda c: MIX(c)["rot"].update(dims=5), 8),
    (lambda c: MIX(c)["rot"]["scaling"].update(factor=0), 8), (lambda c: MIX(c)["rot"]["scaling"].pop("slow"), 8), (lambda c: MLP(c).update(kind="sparse"), 7),
    (lambda c: MLP(c).pop("expert"), 8), (lambda c: MLP(c)["router"].update(experts=7), 8), (lambda c: MLP(c)["router"].update(top=5), 8), (lambda c: MLP(c)["router"].pop("scale"), 8),
    (lambda c: MLP(c)["router"]["groups"].update(keep=4), 8), (lambda c: MLP(c)["shared"].pop("ff"), 8), (lambda c: c["layers"][1]["mixer"].pop("width"), 8),
    (lambda c: c["layers"][3].update(weights_of=3), 8), (lambda c: c["layers"][3].update(weights_of=4), 8), (lambda c: c["layers"][3].update(weights_of=2), 8),
    (lambda c: c["layers"][3].update(weights_of=0.5), 8), (lambda c: c["layers"][1].update(weights_of=3), 8)])
def test_registry_refuses_what_it_cannot_run(change, status):
    c = copy.deepcopy(CFG)
    change(c)
    assert set_config(c)[0] == status


def test_absent_groups_shared_expert_scaling_and_soft_cap_are_allowed():
    c = copy.deepcopy(CFG)
    MLP(c)["router"].pop("groups")
    MLP(c)["shared"] = None
    MIX(c)["rot"].pop("scaling")
    c.pop("logit_softcap")
    assert set_config(c)[0] == 0


def test_a_borrowing_layer_has_no_tensors():
    names = synth.rukedra_specs(CFG)
    assert not any(n.startswith("l3.") for n in names) and "l1.mix.z.b" in names and "l1.rg2" not in names and "l2.rg2.b" in names


# ---- the plain statement against closed forms
def plain(cfg=CFG, seed=1):
    return P.PlainRukedra(cfg, {n: synth.rukedra_tensor(n, s, seed) for n, s in synth.rukedra_specs(cfg).items()})


def test_rotation_keeps_scores_relative_and_scales_only_slow_pairs():
    f, one = P.rotation_speeds(16, 1000.0)
    assert one == 1.0 and np.allclose(f, 1000.0 ** (-np.arange(8) / 8))
    g, gain = P.rotation_speeds(16, 1000.0, {"factor": 4.0, "original": 64, "fast": 4.0, "slow": 1.0})
    turns = 64 * f / (2 * np.pi)
    assert np.allclose(g[turns > 4.5], f[turns > 4.5]) and np.allclose(g[turns < 0.3], f[turns < 0.3] / 4.0) and np.isclose(gain, 1 + 0.1 * np.log(4))
    assert np.all(g <= f) and np.all(g >= f / 4.0)
    r = np.random.default_rng(0)
    q, k = r.standard_normal((2, 16))
    dots = [P.rotate_pairs(q, 9 + s, g, gain) @ P.rotate_pairs(k, 2 + s, g, gain) for s in (0, 5, 300)]
    assert np.allclose(dots, dots[0])
    assert np.allclose(P.rotate_pairs(q, 0, g, gain), q * gain)
    u = P.rotate_pairs(np.array([1.0, 0.0, 0.0, 0.0]), 1, np.array([np.pi / 2, 0.1]), 1.0)
    assert np.allclose(u, [0, 1, 0, 0])                      # neighbours turn together


def test_grouped_norm_has_unit_parts():
    x = np.random.default_rng(1).standard_normal(30) * np.repeat([1.0, 50.0, 0.01], 10)
    y = P.grouped_rms(x, np.ones(30), 3, 0.0).reshape(3, 10)
    assert np.allclose(np.mean(y * y, axis=1), 1.0)
    assert not np.allclose(P.grouped_rms(x, np.ones(30), 1, 0.0), y.reshape(-1))


def test_attend_window_and_equal_scores():
    r = np.random.default_rng(2)
    k, v, q = r.standard_normal((9, 2, 4)), r.standard_normal((9, 2, 3)), r.standard_normal((2, 4))
    assert np.allclose(P.attend(q, k, v, 0.7, 1), v[8])
    assert np.allclose(P.attend(q, k, v, 0.0), v.mean(0))
    assert np.allclose(P.attend(q, k, v, 0.0, 4), v[5:].mean(0))
    assert np.allclose(P.attend(q, k, v, 0.7, 40), P.attend(q, k, v, 0.7))


def test_gelu_against_its_limits():
    z = np.array([-9.0, -1.0, 0.0, 1.0, 9.0])
    y = P.gelu_tanh(z)
    assert np.allclose(y[[0, 2, 4]], [0.0, 0.0, 9.0], atol=1e-9) and np.allclose(y[[1, 3]], [-0.158655, 0.841345], atol=3e-4)


def test_min_gru_is_a_weighted_sum_of_candidates():
    r = np.random.default_rng(4)
    z, u = r.standard_normal((2, 6, 5))
    S = np.zeros(5)
    for t in range(6):
        S = P.min_gru_token(S, z[t], u[t], 0.3, -0.2)
    g, v = P.sigmoid(z + 0.3), u - 0.2
    c = np.where(v >= 0, v + 0.5, P.sigmoid(v))
    assert np.allclose(S, sum(g[t] * c[t] * np.prod(1 - g[t + 1:], axis=0) for t in range(6)))
    assert np.all(c > 0) and np.isclose(P.min_gru_token(np.zeros(1), np.array([99.0]), np.zeros(1), 0, 0)[0], 0.5)


def test_choice_of_experts_by_groups():
    z = np.array([3.0, -1.0, 2.5, 2.4, -2.0, 2.9])          # groups of two: (3, -1), (2.5, 2.4), (-2, 2.9)
    pick, w = P.choose_experts(z, 2, 3, 1, 2.0)
    s = P.sigmoid(z)
    assert list(pick) == [2, 3] and np.allclose(w, 2.0 * s[[2, 3]] / (s[2] + s[3]))      # the best single expert's group loses
    assert list(P.choose_experts(z, 2, 3, 3, 1.0)[0]) == [0, 5] and list(P.choose_experts(z, 2, 1, 1, 1.0)[0]) == [0, 5]
    assert np.isclose(P.choice_margin(z, 2, 1, 1), s[5] - s[2])


def test_portions_and_soft_cap_of_the_plain_model():
    m = plain()
    t = [int(x) for x in np.random.default_rng(5).integers(0, 53, 20)]
    whole = m.forward(t, m.new_state())
    st = m.new_state()
    parts = np.concatenate([m.forward(t[:7], st), m.forward(t[7:], st)])
    assert np.array_equal(whole, parts) and np.max(np.abs(whole)) < 7.0
    free = P.PlainRukedra(dict(CFG, logit_softcap=None), m.w)
    assert np.allclose(7.0 * np.tanh(free.forward(t, free.new_state()) / 7.0), whole)
