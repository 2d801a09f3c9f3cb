"""Rukedra models on the GPU against the plain statement of their mechanisms (plain_rukedra.py): every mixer and feed-forward alone
and together, prompts against decoding, portions, sequences after and beside one another, window edges, far keys, long decoding,
shared tensors, generation.  Errors are root mean square over the vocabulary, relative to the logits' own."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import layered_session as S
import plain_rukedra as P
import tl_b200 as tl
from layered_session import decode, err, greedy, run_portions, toks
from tl_b200 import synth

pytestmark = pytest.mark.gpu
TOL = {True: 2e-5, False: 2.5e-2}           # f32; bf16 operands
BOTH = pytest.mark.parametrize("f32", [True, False], ids=["f32", "bf16"])
YARN = {"factor": 3.0, "original": 40, "fast": 8.0, "slow": 0.5}


def latent(heads=3, dim=20, rot_dim=12, vdim=28, kv_rank=44, q_rank=36, window=19, scale=0.2, base=700.0, scaling=YARN):
    """q_rank None: direct queries, no window, no output gate."""
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "rot": {"base": base, "dims": rot_dim}}
    if scaling:
        m["rot"]["scaling"] = dict(scaling)
    if q_rank is None:
        return {"type": "latent_attention_2", "mixer": m}
    m["q_rank"], m["mask"] = q_rank, {"size": window}
    return {"type": "latent_attention", "mixer": m}


def direct(**kw):
    return latent(q_rank=None, **kw)


def gru(width=52):
    return {"type": "mingru", "mixer": {"width": width}}


def dense(ff=60):
    return {"kind": "dense", "ff": ff}


def moe(experts=10, top=3, ff=28, groups=(5, 3), scale=1.7, shared=36):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if groups:
        f["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def config(layers, width=72, vocab=131, eps=1e-5, groups=3, cap=9.0):
    """layers: (mixer, feed-forward or None) pairs, or a number: a layer with that layer's tensors."""
    out = []
    for l in layers:
        out.append(dict(copy.deepcopy(out[l]), weights_of=l) if isinstance(l, int) else dict(copy.deepcopy(l[0]), mlp=copy.deepcopy(l[1])))
    return {"architecture": "Rukedra", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups}, "logit_softcap": cap, "layers": out}


MIXED = [(direct(), dense()), (latent(), moe()), (gru(), dense(44)), (gru(20), None), (direct(heads=5, dim=40, rot_dim=8, vdim=72, kv_rank=72, scale=0.14), moe(8, 2, 20, None, 1.0, None)),
         (latent(heads=2, dim=64, rot_dim=32, vdim=40, kv_rank=24, q_rank=20, window=70, scale=0.1), None), 2, 1]


class Model(S.Model):
    def __init__(self, cfg, seed=1, edit=None):
        super().__init__(cfg, synth.rukedra_specs(cfg), synth.rukedra_tensor, P.PlainRukedra, seed, edit)

    def sure(self, n, seed=0, margin=0.03):
        """n tokens whose choices of experts are all clear ones, so that rounding cannot turn one, and their logits."""
        draw = np.random.default_rng(seed)
        st, out, want = self.plain.new_state(), [], []
        while len(out) < n:
            t = int(draw.integers(0, self.cfg["vocab"]))
            trial = {"pos": st["pos"], "layers": [{k: list(v) if isinstance(v, list) else v for k, v in l.items()} for l in st["layers"]]}
            self.plain.margins.clear()
            lg = self.plain.token(t, trial)
            if all(m > margin for m in self.plain.margins):
                st = trial
                out.append(t)
                want.append(lg)
        return out, np.stack(want)


def close(a, b, f32):
    """With bf16 operands the middle row's error is what the roundings usually come to, and a few rows of a deep model are less well
    conditioned: the plain statement with its operands rounded to bf16 reaches 0.04 to 0.09 on these models, at a median of 0.009."""
    e = S.row_errors(a, b)
    return float(np.max(e)) < (TOL[True] if f32 else 8e-2) and (f32 or len(e) < 20 or float(np.median(e)) < 1.5e-2)


# ---- mechanisms alone, at sizes that are multiples of nothing and at ones that coincide or are 1
MIXERS = {
    "latent": latent(), "latent_window_1": latent(window=1), "latent_wide_window": latent(window=100000), "latent_plain_angles": latent(scaling=None),
    "latent_factor_1": latent(scaling=dict(YARN, factor=1.0)), "latent_narrow_ramp": latent(scaling={"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}),
    "latent_tiny": latent(heads=1, dim=1, rot_dim=2, vdim=1, kv_rank=1, q_rank=1, window=6, scale=1.0), "latent_17_heads": latent(heads=17, dim=8, rot_dim=4, vdim=5, kv_rank=16, window=64),
    "latent_equal": latent(heads=4, dim=32, rot_dim=32, vdim=32, kv_rank=32, q_rank=32, window=33, scale=0.125),
    "latent_80": latent(heads=2, dim=64, rot_dim=16, vdim=64, kv_rank=48, window=66, scale=0.1), "latent_84_odd": latent(heads=3, dim=70, rot_dim=14, vdim=66, kv_rank=47, q_rank=35, window=90, scale=0.1), "latent_rank_130": latent(heads=2, kv_rank=130, window=90),
    "direct": direct(), "direct_one_head": direct(heads=1), "direct_192": direct(heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=200, scale=0.07),
    "direct_170": direct(heads=2, dim=130, rot_dim=40, vdim=100, kv_rank=88, scale=0.07), "direct_256": direct(heads=2, dim=200, rot_dim=56, vdim=150, kv_rank=64, scale=0.06),
    "direct_300": direct(heads=2, dim=280, rot_dim=20, vdim=270, kv_rank=40, scale=0.06), "direct_rank_300": direct(heads=3, kv_rank=300), "direct_rank_600": direct(heads=2, kv_rank=600, rot_dim=10),
    "direct_odd": direct(heads=3, dim=13, rot_dim=6, vdim=11, kv_rank=21, scale=0.3, base=33.0),
    "gru": gru(), "gru_one": gru(1), "gru_33": gru(33), "gru_300": gru(300)}


@BOTH
@pytest.mark.parametrize("name", sorted(MIXERS))
def test_mixer_alone(name, f32):
    if not f32 and name == "latent_tiny":
        pytest.skip("one number over its own root mean square is its sign: a rounding that crosses zero flips it")
    m = Model(config([(MIXERS[name], None)]), seed=3)
    t = toks(150)
    want = m.ref(t)
    d = m.dec(f32)
    assert close(d.prefill_logits(t[:139]), want[:139], f32)
    assert close(decode(d, t[139:], 139), want[139:], f32)
    assert close(decode(m.dec(f32), t[:24], 0), want[:24], f32)
    assert close(run_portions(m.dec(f32), t[:90], [2, 7, 30]), want[:90], f32)


@BOTH
@pytest.mark.parametrize("sizes", [dict(dim=64, rot_dim=16, vdim=64, kv_rank=48), dict(dim=128, rot_dim=60, vdim=101, kv_rank=72), dict(dim=12, rot_dim=10, vdim=9, kv_rank=20)], ids=["80", "188", "22"])
def test_long_portions_behind_a_window(sizes, f32):
    """Portions whose window starts well behind the first cache row."""
    m = Model(config([(latent(heads=2, window=66, scale=0.1, **sizes), None)]), seed=6)
    t = toks(460)
    want = m.ref(t)
    for portions in ([200, 130, 65], [129, 70], [300, 100, 2]):
        assert close(run_portions(m.dec(f32, max_seq=460), t, portions), want, f32), portions


FFNS = {
    "dense": dense(), "dense_1": dense(1), "dense_1030": dense(1030), "dense_12200": dense(12200), "moe": moe(), "moe_no_groups": moe(groups=None), "moe_one_group": moe(groups=(1, 1)),
    "moe_groups_of_one": moe(6, 2, groups=(6, 4)), "moe_keeps_all": moe(8, 3, groups=(4, 4)), "moe_keeps_one": moe(14, 4, groups=(2, 1)), "moe_top_1": moe(7, 1, groups=None),
    "moe_every_expert": moe(4, 4, groups=(2, 2)), "moe_one_expert": moe(1, 1, groups=None), "moe_no_shared": moe(shared=None), "moe_sizes": moe(40, 6, 260, (8, 3), 2.5, 300), "moe_48_kB": moe(7, 6, 1500, (7, 6), 1.0, 3000), "moe_ff_1": moe(5, 2, 1, None, 1.0, 1)}


@BOTH
@pytest.mark.parametrize("name", sorted(FFNS))
def test_feed_forward_alone(name, f32):
    m = Model(config([(gru(16), FFNS[name])]), seed=4)
    t, want = m.sure(80)
    d = m.dec(f32)
    assert close(d.prefill_logits(t[:61]), want[:61], f32)
    assert close(decode(d, t[61:], 61), want[61:], f32)
    assert close(run_portions(m.dec(f32), t, [2, 3]), want, f32)


@BOTH
@pytest.mark.parametrize("width,groups,vocab,eps,cap", [(72, 1, 131, 1e-5, 3.0), (33, 11, 7, 1e-2, 50.0), (256, 2, 1000, 1e-6, 30.0), (500, 50, 129, 1e-5, 1.0), (21, 3, 40, 1e-5, None), (1032, 4, 64, 1e-5, 20.0)])
def test_norms_gates_and_soft_cap(width, groups, vocab, eps, cap, f32):
    m = Model(config([(direct(), dense()), (latent(), None), (gru(), moe())], width=width, groups=groups, vocab=vocab, eps=eps, cap=cap), seed=5)
    t, want = m.sure(40)
    d = m.dec(f32)
    assert close(d.prefill_logits(t[:33]), want[:33], f32)
    assert close(decode(d, t[33:], 33), want[33:], f32)
    layers = [[] for _ in m.cfg["layers"]]
    m.plain.forward(t, m.plain.new_state(), layers)
    x = layers[-1][-1]
    assert np.allclose(d.hidden(), x, atol=(1e-4 if f32 else 6e-2) * np.max(np.abs(x)))


@BOTH
def test_a_width_beyond_the_registers_of_a_launch(f32):
    m = Model(config([(gru(16), None), 0], width=4224, groups=3, vocab=40), seed=5)
    t = toks(14, 40)
    want = m.ref(t)
    d = m.dec(f32)
    assert close(d.prefill_logits(t[:9]), want[:9], f32)
    assert close(decode(d, t[9:], 9), want[9:], f32)


def test_the_gate_and_the_norms_matter():
    """Dropping a mechanism moves the plain logits far beyond the tolerances above."""
    m = Model(config([(latent(), moe())]), seed=5)
    t = toks(30)
    want = m.ref(t)
    for change in ({"l0.rg1": 0.0, "l0.rg1.b": 9.0}, {"l0.rg2": 0.0, "l0.rg2.b": 9.0}, {"l0.norm1b": 1.0}, {"l0.norm2b": 1.0}, {"l0.mix.g": 0.0}, {"l0.mix.dq.norm": 1.0},
                   {"l0.mix.dkv.norm": 1.0}, {"l0.mlp.shared.sg": 0.0}):
        w = dict(m.plain.w)
        for n, v in change.items():
            w[n] = np.full_like(w[n], v)
        other = P.PlainRukedra(m.cfg, w)
        assert err(other.forward(t, other.new_state()), want) > 0.05, change


# ---- whole models
@BOTH
def test_prompt_decoding_and_portions_agree(f32):
    m = Model(config(MIXED), seed=7)
    t, want = m.sure(210)
    assert close(m.dec(f32).prefill_logits(t), want, f32)
    assert close(decode(m.dec(f32), t[:120], 0), want[:120], f32)
    for sizes in ([2], [3, 2], [64], [17, 2, 64, 1, 5], [16], [15, 33], [128, 2]):
        assert close(run_portions(m.dec(f32), t[:160], sizes), want[:160], f32), sizes


@BOTH
def test_sequences_one_after_the_other_leave_nothing_behind(f32):
    m = Model(config(MIXED), seed=8)
    (a, want_a), (b, want_b) = m.sure(150, seed=1), m.sure(60, seed=2)
    d = m.dec(f32)
    first = run_portions(d, a, [70, 2, 1])
    assert close(first, want_a, f32)
    assert close(run_portions(d, b, [1, 5, 20]), want_b, f32)               # starts with a decode step at position 0
    assert np.array_equal(first, run_portions(d, a, [70, 2, 1]))


@BOTH
def test_batch_of_unequal_sequences_against_each_alone(f32):
    m = Model(config(MIXED), seed=9)
    lens, again = [90, 3, 41, 66], 37
    d = m.dec(f32, batch=len(lens))
    seqs = [m.sure(n + 35, seed=20 + i) for i, n in enumerate(lens)]
    for i, n in enumerate(lens):
        assert close(run_portions(d, seqs[i][0][:n], [25, 2], seq=i), seqs[i][1][:n], f32)

    def run(steps, at):
        got = []
        for s in range(steps):
            d.step_batch([t[p + s] for (t, _), p in zip(seqs, at)], [p + s for p in at], read=False)
            got.append(d.logits_batch())
        for i, p in enumerate(at):
            assert close(np.stack([g[i] for g in got]), seqs[i][1][p:p + steps], f32), (i, p)

    run(30, lens)
    # one slot is freed and used again while the others go on
    seqs[1] = m.sure(again + 5, seed=77)
    assert close(run_portions(d, seqs[1][0][:again], [again], seq=1), seqs[1][1][:again], f32)
    run(5, [again if i == 1 else n + 30 for i, n in enumerate(lens)])


@BOTH
def test_layers_with_another_layers_tensors(f32):
    """A layer may use the tensors of one before, of one behind, or of one that itself borrows; the state is its own."""
    cfg = config([(latent(), dense()), (gru(), None), 0, 1, (direct(), moe())])
    cfg["layers"].insert(0, dict(copy.deepcopy(cfg["layers"][4]), weights_of=5))
    for l in cfg["layers"][3:5]:
        l["weights_of"] += 1
    cfg["layers"].append(dict(copy.deepcopy(cfg["layers"][3]), weights_of=3))
    m = Model(cfg, seed=10)
    t, want = m.sure(90)
    d = m.dec(f32)
    assert close(d.prefill_logits(t[:70]), want[:70], f32)
    assert close(decode(d, t[70:], 70), want[70:], f32)
    alone = copy.deepcopy(cfg)
    for l in alone["layers"]:
        l.pop("weights_of", None)
    own = Model(alone, seed=10)                         # tensors of its own for every layer: another model
    assert err(own.ref(t), want) > 0.05


# ---- edges: one key stands out so far that seeing it or not changes everything
def standout(lay, gain, width=64):
    """Token 5's latent answers the query of every token with a score about `gain` above the others; its value is another one."""
    cfg = config([(dict(lay, mixer=dict(lay["mixer"], scale=1.0)), None)], width=width, groups=2, vocab=40, cap=30.0)
    x = lay["mixer"]
    hd, D, R = x["dim"] + x["rot_dim"], x["dim"], x["kv_rank"]

    def edit(v):
        e = v["embed"]
        e[:] *= 0.3
        e[:, 0] = 0.0
        e[:, 1] = 3.0                                    # every query's part in common
        e[5, 0] = 8.0
        v["l0.norm1"][:] = 1.0
        v["l0.mix.dkv"][:, 0] = 0.0
        v["l0.mix.dkv"][0] = 0.0
        v["l0.mix.dkv"][0, 0] = 5.0                      # token 5's latent is little but its first element, about sqrt(R)
        v["l0.mix.dkv.norm"][:] = 1.0
        v["l0.mix.dkv"][R:] *= 0.1
        v["l0.mix.uk"][:] *= 0.1
        v["l0.mix.uk"][0::D, 0] = gain / np.sqrt(R)
        if "l0.mix.uq" in v:
            K = x["q_rank"]
            v["l0.mix.dq"][:] *= 0.05
            v["l0.mix.dq"][0] = 0.0
            v["l0.mix.dq"][0, 1] = 1.0
            v["l0.mix.dq.norm"][:] = 1.0
            v["l0.mix.uq"][:] *= 0.1
            v["l0.mix.uq"][0::hd, :] = 0.0
            v["l0.mix.uq"][0::hd, 0] = 1.0 / np.sqrt(K)
        else:
            v["l0.mix.q"][:] *= 0.1
            v["l0.mix.q"][0::hd, :] = 0.0
            v["l0.mix.q"][0::hd, 1] = 0.4
    return Model(cfg, seed=11, edit=edit)


@BOTH
@pytest.mark.parametrize("sizes", [dict(dim=40, rot_dim=8, vdim=32, kv_rank=48), dict(dim=96, rot_dim=32, vdim=96, kv_rank=64), dict(dim=128, rot_dim=64, vdim=128, kv_rank=80)], ids=["48", "128", "192"])
@pytest.mark.parametrize("window", [2, 16, 63, 64, 65, 128, 130])
def test_window_edge_in_prompts_portions_and_decoding(window, sizes, f32):
    m = standout(latent(heads=2, window=window, **sizes), gain=7.0)
    n = 2 * window + 80
    for place in (0, 7, 63, 64):
        t = [(3 + i) % 5 for i in range(n)]
        t[place] = 5
        want = m.ref(t)
        inside, outside = place + window - 1, place + window
        moved = err(want[outside], want[inside])
        assert moved > 0.2, "the input does not show the edge: %g" % moved
        got = m.dec(f32, max_seq=512).prefill_logits(t)
        cut = max(1, inside - 2)
        d = m.dec(f32, max_seq=512)
        d.prefill_logits(t[:cut], want=[])
        dec = decode(d, t[cut:outside + 3], cut)
        d = m.dec(f32, max_seq=512)
        d.prefill_logits(t[:cut], want=[])
        por = run_portions(d, t[:outside + 3], [2, 4], at=cut)
        tol = 1e-4 if f32 else 3e-2
        for p in (place, place + 1, inside - 1, inside, outside, outside + 1, n - 1):
            if p < n:
                assert err(got[p], want[p]) < tol, (window, place, p)
            if cut <= p < outside + 3:
                assert err(dec[p - cut], want[p]) < tol, (window, place, p)
                assert err(por[p - cut], want[p]) < tol, (window, place, p)


@BOTH
def test_far_key_behind_hundreds_of_others(f32):
    """One key far back holds half the weight: a lost row, split or tile would show."""
    m = standout(direct(heads=2, dim=40, rot_dim=16, vdim=48, kv_rank=64, scaling=dict(YARN, original=300)), gain=7.0)
    t = [(3 + i) % 5 for i in range(700)]
    t[2] = 5
    want = m.ref(t)
    without = m.ref([t[0], t[1], 3] + t[3:])
    assert err(without[699], want[699]) > 0.2
    d = m.dec(f32, max_seq=1024)
    got = d.prefill_logits(t[:640])
    rows = [2, 3, 63, 64, 65, 127, 128, 300, 511, 512, 513, 639]
    tol = 1e-4 if f32 else 3e-2
    assert err(got[rows], want[rows]) < tol
    assert err(decode(d, t[640:670], 640), want[640:670]) < tol
    assert err(run_portions(d, t, [2, 3], at=670), want[670:]) < tol


@BOTH
def test_state_remembers_a_far_token(f32):
    """A gate that is nearly closed: what the first token left still moves the logits hundreds of tokens later."""
    def edit(v):
        v["l0.mix.z"][:] *= 0.3
        v["l0.mix.z.b"][:] = -7.0
        v["l0.mix.z"][:, 0] = 6.0
        v["embed"][:, 0] = 0.0
        v["embed"][7:9, 0] = 6.0                          # tokens 7 and 8 open it
    m = Model(config([(gru(40), None)], width=64, groups=1, vocab=40), seed=12, edit=edit)
    t = [7] + [(3 + i) % 6 for i in range(600)]
    want = m.ref(t)
    assert err(m.ref([8] + t[1:])[600], want[600]) > 1e-2
    d = m.dec(f32, max_seq=700)
    assert err(run_portions(d, t[:560], [100, 2, 33]), want[:560]) < TOL[f32]
    assert err(decode(d, t[560:], 560), want[560:]) < TOL[f32]


@BOTH
def test_long_decoding(f32):
    m = Model(config([(direct(), dense()), (latent(window=50), None), (gru(), dense())]), seed=13)
    t = toks(400)
    assert close(decode(m.dec(f32, max_seq=400), t, 0), m.ref(t), f32)


@BOTH
def test_prompt_longer_than_a_chunk(f32):
    """2,100 tokens: the session cuts a prompt after 2,048."""
    m = Model(config([(direct(heads=2, dim=64, rot_dim=16, vdim=32, kv_rank=24), None), (latent(heads=1, window=300), None), (gru(16), None)], width=32, groups=2), seed=14)
    t = toks(2100)
    want = m.ref(t)
    rows = [0, 1, 2046, 2047, 2048, 2049, 2099]
    assert err(m.dec(f32, max_seq=2200).prefill_logits(t, want=rows), want[rows]) < TOL[f32]
    d = m.dec(f32, max_seq=2200)
    d.prefill_logits(t[:2047], want=[])
    assert err(d.prefill_logits(t[2047:], 2047), want[2047:]) < TOL[f32]


# ---- generation through the session's own entry points
def test_greedy_generation():
    m = Model(config(MIXED), seed=15)
    prompt = toks(45, seed=5)
    want, gap = greedy(m, prompt, 24)
    assert gap > 1e-4                                     # no tie that rounding could turn
    d = m.dec(True)
    first = d.prefill(prompt)
    assert [first] + d.generate(first, 45, 23) == want
    d2 = m.dec(True)
    tok, got = d2.prefill(prompt), []
    for i in range(24):
        got.append(tok)
        tok = d2.step(tok, 45 + i)
    assert got == want


def test_greedy_generation_of_a_batch():
    m = Model(config(MIXED), seed=15)
    prompts = [toks(45, seed=5), toks(12, seed=6), toks(70, seed=7)]
    d = m.dec(True, batch=3)
    firsts = [d.prefill_seq(i, p) for i, p in enumerate(prompts)]
    out = d.generate_batch(firsts, [len(p) for p in prompts], 11)
    for i, p in enumerate(prompts):
        want, gap = greedy(m, p, 12)
        assert gap > 1e-4
        assert [firsts[i]] + [int(t) for t in out[:, i]] == want


def test_sampled_generation_is_the_sampler_on_each_step():
    m = Model(config(MIXED), seed=16)
    prompt = toks(20, seed=9)
    d = m.dec(True)
    first = d.prefill(prompt)
    got = d.generate_sampled(first, 20, 12, 0.8, 20, 0.9, seed=4)
    d2 = m.dec(True)
    d2.prefill(prompt)
    tok = first
    for i in range(12):
        d2.step(tok, 20 + i, read=False)
        tok = tl.Tensor.from_numpy(d2.logits()).sample_top_k_top_p(0.8, 20, 0.9, tl.rng_uniform(4, i)).item_i64()
        assert tok == got[i], i


def test_step_statistics():
    """A step reads the experts it uses, a borrowed layer's tensors once per layer, and the window's part of a cache."""
    W, V = 72, 131
    cfg = config([(latent(), moe()), (gru(), None), 0])
    shapes = synth.rukedra_specs(cfg)
    st = Model(cfg).dec(False).stats(100)
    f = cfg["layers"][0]["mlp"]
    size = lambda n: int(np.prod(shapes[n])) * (2 if len(shapes[n]) == 2 else 4)
    layer = [sum(size(n) for n in shapes if n.startswith("l%d." % i) and ".mlp.e" not in n) for i in (0, 1)]
    experts = f["router"]["top"] * 3 * f["expert"]["ff"] * W * 2
    assert st["weight_bytes"] == 2 * (layer[0] + experts) + layer[1] + (V + 1) * W * 2 + W * 4
    assert st["kv_bytes"] == 2 * 19 * (44 + 12) * 2 + 2 * 52 * 4 and st["kernels_per_step"] == 9 + 3 + 9 + 1 + 1


def test_model_folder_loads_to_the_same_model(tmp_path):
    m = Model(config(MIXED), seed=17)
    synth.write_model_dir(tmp_path / "m", m.cfg, m.bits)
    w = tl.TensorMap.load_dir(tmp_path / "m")
    assert w.meta_string("general.architecture") == "Rukedra" and w.decoder_cfg()["n_layers"] == len(MIXED)
    t = toks(50)
    a = tl.Decoder(None, w, max_seq=64, f32=True).prefill_logits(t)
    assert np.array_equal(a, m.dec(True, max_seq=64).prefill_logits(t))


def test_missing_or_misshapen_tensors_are_refused():
    cfg = config(MIXED)
    cut = lambda n: lambda b: b.update({n: b[n][:-1]})
    for change, code in ((lambda b: b.pop("l1.mix.dq.norm"), 8), (lambda b: b.pop("l0.mix.q"), 8), (lambda b: b.pop("l2.mix.z.b"), 8), (lambda b: b.pop("l1.mlp.e9.up"), 8),
                         (lambda b: b.pop("l3.rg1.b"), 8), (cut("l1.mlp.router"), 1), (cut("l0.mix.uk"), 1), (cut("l4.norm2b"), 1), (cut("l2.mix.o"), 1)):
        bits = synth.rukedra_tensors(cfg, 1)
        change(bits)
        w = tl.TensorMap.new()
        for n, b in bits.items():
            w.add(n, synth.BF16, b.shape, np.ascontiguousarray(b))
        w.set_config(json.dumps(cfg))
        with pytest.raises(tl.TlbError) as e:
            tl.Decoder(None, w, max_seq=32)
        assert e.value.code == code


def test_command_line_generates_from_a_folder(tmp_path, capsys):
    from tl_b200 import generate
    m = Model(config(MIXED), seed=15)
    synth.write_model_dir(tmp_path / "m", m.cfg, m.bits)
    prompt = toks(45, seed=5)
    generate.main(["--model", str(tmp_path / "m"), "--tokens", ",".join(map(str, prompt)), "--f32", "-n", "12"])
    assert [int(x) for x in capsys.readouterr().out.split(",")] == greedy(m, prompt, 12)[0]


def test_trace_replay(tmp_path):
    """bin/trace_run: the logits of the wanted tokens, whatever the portions, for requests one after the other."""
    m = Model(config(MIXED), seed=18)
    synth.write_model_dir(tmp_path / "m", m.cfg, m.bits)
    (a, wa), (b, wb) = m.sure(30, seed=1), m.sure(9, seed=2)
    steps = [([("a", a[:20], [0, 19])], []), ([("a", a[20:22], [])], []), ([("a", a[22:23], [0])], []), ([("a", a[23:], [6, 2])], ["a"]),
             ([("b", b[:1], [0])], []), ([("b", b[1:], [7])], ["b"])]
    want = [wa[[0, 19]], None, wa[[22]], wa[[29, 25]], wb[[0]], wb[[8]]]
    text = "".join(json.dumps({"step": i, "entries": [{"id": r, "tokens": t, "want": w} for r, t, w in e], "end": end}) + "\n" for i, (e, end) in enumerate(steps))
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(out), "--max-tokens", "30"],
                           input=text, capture_output=True, text=True, timeout=300)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done %d" % i for i in range(len(steps))]
        for i, w in enumerate(want):
            f = out / ("%d.f32" % i)
            assert f.exists() == (w is not None)
            if w is not None:
                assert close(np.frombuffer(f.read_bytes(), dtype="<f4").reshape(-1, m.cfg["vocab"]), w, dtype == "float32")
