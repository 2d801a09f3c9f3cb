"""Models described by a config.json on the GPU against the plain statement of their mechanisms (plain_layers.py): every mixer
alone and together, prompts against decoding, portions, sequences after and beside one another, window edges, long decoding,
generation.  Errors are root mean square over the vocabulary, relative to the logits' own."""
import copy
import json

import numpy as np
import pytest

import layered_session as S
import plain_layers as P
import tl_b200 as tl
from layered_session import decode, err, greedy, run_portions, toks
from tl_b200 import synth

pytestmark = pytest.mark.gpu
TOL = {True: 2e-5, False: 2.5e-2}           # f32; bf16 operands
BOTH = pytest.mark.parametrize("f32", [True, False], ids=["f32", "bf16"])


def attention(heads=6, kv=3, dim=24, vdim=40, window=19, scale=0.2):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window}}}


def retention(heads=3, dim=24, vdim=40, dims=16, base=1000.0, decay=None):
    d = decay if decay is not None else [1.0 - 2.0 ** (-2 - 2 * i) for i in range(heads)]
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": dims}, "decay": d}}


def delta(heads=3, dim=28):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}}


def config(layers, width=72, ff=100, vocab=131, eps=1e-5, mlps=None):
    out = []
    for i, l in enumerate(layers):
        has = ff and (mlps is None or mlps[i])
        out.append(dict(copy.deepcopy(l), mlp={"kind": "dense", "ff": ff} if has else None))
    return {"architecture": "Mukutar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": out}


MIXED = [retention(), attention(), delta(), attention(heads=4, kv=1, dim=40, vdim=24, window=70), retention(heads=2, dim=40, vdim=16, dims=40), delta(heads=2, dim=64)]


class Model(S.Model):
    def __init__(self, cfg, seed=1, rank=11, edit=None):
        super().__init__(cfg, synth.mukutar_specs(cfg, rank), synth.mukutar_tensor, P.Plain, seed, edit)


def close(a, b, f32):
    """Every row within the tolerance; with bf16 operands all but 3 % of them (at least one): a head's output over its own root mean
    square jumps where it crosses zero - on a sequence's first token it is little more than the sign of one dot product."""
    e = S.row_errors(a, b)
    return int(np.sum(e >= TOL[f32])) <= (0 if f32 else max(1, int(0.03 * len(e))))


# ---- mechanisms alone, at sizes that are multiples of nothing and at ones that coincide or are 1
ALONE = {
    "attention": attention(), "attention_window_1": attention(window=1), "attention_one_head": attention(heads=1, kv=1, dim=1, vdim=1, window=6),
    "attention_mha": attention(heads=5, kv=5, dim=32, vdim=32, window=33), "attention_mqa": attention(heads=7, kv=1, dim=18, vdim=6, window=64),
    "attention_wide_window": attention(window=100000), "attention_96": attention(heads=2, kv=1, dim=96, vdim=96, window=40),
    "attention_128_112": attention(heads=3, kv=1, dim=128, vdim=112, window=130, scale=0.09), "attention_72_100": attention(heads=2, kv=2, dim=72, vdim=100, window=61, scale=0.1),
    "attention_136": attention(heads=2, kv=1, dim=136, vdim=50, window=77, scale=0.1), "attention_256": attention(heads=2, kv=1, dim=256, vdim=200, window=50, scale=0.06),
    "retention": retention(), "retention_one": retention(heads=1, dim=2, vdim=1, dims=2, decay=[0.5]), "retention_fast": retention(heads=2, decay=[0.01, 1.0]),
    "retention_128": retention(heads=2, dim=128, vdim=128, dims=64), "retention_odd": retention(heads=3, dim=23, vdim=37, dims=10),
    "retention_160": retention(heads=1, dim=160, vdim=70, dims=160), "retention_256": retention(heads=1, dim=250, vdim=33, dims=96),
    "delta": delta(), "delta_one": delta(heads=1, dim=1), "delta_32": delta(heads=4, dim=32), "delta_odd": delta(heads=2, dim=37), "delta_96": delta(heads=1, dim=96),
    "delta_128": delta(heads=2, dim=128), "delta_192": delta(heads=1, dim=192), "delta_224": delta(heads=1, dim=224), "delta_256": delta(heads=1, dim=256)}


@BOTH
@pytest.mark.parametrize("name", sorted(ALONE))
def test_mixer_alone(name, f32):
    if not f32 and name in ("delta_one", "retention_one"):
        pytest.skip("one value channel over its own root mean square is its sign: a rounding that crosses zero flips it")
    m = Model(config([ALONE[name]], ff=0), seed=3, rank=1 if name.endswith("one") else 11)
    t = toks(150)
    want = m.ref(t)
    d = m.dec(f32)
    got = d.prefill_logits(t[:139])
    assert close(got, want[:139], f32)
    assert close(decode(d, t[139:], 139), want[139:], f32)
    d2 = m.dec(f32)
    assert close(decode(d2, t[:24], 0), want[:24], f32)


@BOTH
@pytest.mark.parametrize("width,ff,vocab,eps", [(72, 100, 131, 1e-5), (33, 1, 7, 1e-2), (256, 640, 1000, 1e-6), (520, 2051, 129, 1e-5)])
def test_norms_feed_forward_and_scales(width, ff, vocab, eps, f32):
    """Layer scales, norms around zero and PolyNorm with a large eps as well; the layer in the middle has no feed-forward."""
    m = Model(config([attention(), delta(), retention()], width=width, ff=ff, vocab=vocab, eps=eps, mlps=[1, 0, 1]), seed=5)
    t = toks(40, vocab)
    want = m.ref(t)
    d = m.dec(f32)
    assert close(d.prefill_logits(t[:33]), want[:33], f32)
    assert close(decode(d, t[33:], 33), want[33:], f32)
    assert np.allclose(d.hidden(), m_hidden(m, t), atol=(1e-4 if f32 else 6e-2) * np.max(np.abs(m_hidden(m, t))))


def m_hidden(m, t):
    layers = [[] for _ in m.cfg["layers"]]
    m.plain.forward(t, m.plain.new_state(), layers)
    return layers[-1][-1]


# ---- whole models
@BOTH
def test_prompt_decoding_and_portions_agree(f32):
    m = Model(config(MIXED), seed=7)
    t = toks(210)
    want = m.ref(t)
    d = m.dec(f32)
    whole = d.prefill_logits(t)
    assert err(whole, want) < TOL[f32]
    one = decode(m.dec(f32), t[:120], 0)
    assert err(one, want[:120]) < TOL[f32]
    for sizes in ([2], [3, 2], [64], [17, 2, 64, 1, 5], [16], [15, 33], [128, 2]):
        got = run_portions(m.dec(f32), t[:160], sizes)
        assert err(got, want[:160]) < TOL[f32], sizes


@BOTH
def test_sequences_one_after_the_other_leave_nothing_behind(f32):
    m = Model(config(MIXED), seed=8)
    a, b = toks(150, seed=1), toks(60, seed=2)
    d = m.dec(f32)
    first = run_portions(d, a, [70, 2, 1])
    assert err(first, m.ref(a)) < TOL[f32]
    assert err(run_portions(d, b, [1, 5, 20]), m.ref(b)) < TOL[f32]         # starts with a decode step at position 0
    again = run_portions(d, a, [70, 2, 1])
    assert np.array_equal(first, again)


def test_a_sequence_goes_on_only_from_where_it_stands():
    m = Model(config(MIXED), seed=8)
    d = m.dec(True)
    d.prefill(toks(10))
    for call in (lambda: d.step(1, 11), lambda: d.prefill([1, 2], 9), lambda: d.generate(1, 5, 3), lambda: d.prefill_logits([1, 2], 12)):
        with pytest.raises(tl.TlbError):
            call()
    d.step(1, 10)
    d.step(1, 0)
    d.reset_seq()
    d.prefill(toks(4))
    for bad in (lambda: d.prefill_logits([1, 500], 4), lambda: d.prefill_logits([1], 4, want=[1]), lambda: d.prefill(toks(300), 0), lambda: d.kv_write(0, 0, np.zeros((1, 4)), np.zeros((1, 4)))):
        with pytest.raises(tl.TlbError):
            bad()


@BOTH
def test_batch_of_unequal_sequences_against_each_alone(f32):
    m = Model(config(MIXED), seed=9)
    lens = [90, 3, 41, 66]
    d = m.dec(f32, batch=len(lens))
    prompts = [toks(n, seed=20 + i) for i, n in enumerate(lens)]
    follow = [toks(30, seed=40 + i) for i in range(len(lens))]
    for i, p in enumerate(prompts):
        assert err(run_portions(d, p, [25, 2], seq=i), m.ref(p)) < TOL[f32]
    want = [m.ref(p + f)[len(p):] for p, f in zip(prompts, follow)]
    for s in range(30):
        d.step_batch([f[s] for f in follow], [n + s for n in lens], read=False)
        lg = d.logits_batch()
        for i in range(len(lens)):
            assert err(lg[i], want[i][s]) < TOL[f32], (s, i)
    # one slot is freed and used again while the others go on
    p = toks(37, seed=77)
    assert err(run_portions(d, p, [37], seq=1), m.ref(p)) < TOL[f32]
    want1 = m.ref(p + follow[1])[len(p):]
    full = [m.ref(pp + f + f)[len(pp) + 30:] for pp, f in zip(prompts, follow)]
    for s in range(5):
        d.step_batch([f[s] for f in follow], [n + 30 + s if i != 1 else 37 + s for i, n in enumerate(lens)], read=False)
        lg = d.logits_batch()
        for i in range(len(lens)):
            assert err(lg[i], want1[s] if i == 1 else full[i][s]) < TOL[f32], (s, i)


# ---- edges: one key stands out so far that seeing it or not changes everything
def standout(window, heads=2, kv=1, dim=48, vdim=32, r=0.0, sink=None, width=64, gain=6.0):
    """Token 5's key answers every query with a score about `gain` above the others; its value is large."""
    cfg = config([attention(heads=heads, kv=kv, dim=dim, vdim=vdim, window=window, scale=1.0)], width=width, ff=0, vocab=40)

    def edit(v):
        e = v["embed"]
        e[:] *= 0.5
        e[:, 0] = 0.0
        e[5] = 0.0
        e[5, 0] = 8.0
        v["l0.norm1"][:] = 0.0
        v["l0.mix.k"][:, 0] = 0.0
        for n in ("q", "k"):
            v["l0.mix.%s" % n][:] *= 0.1
            v["l0.mix.%s.b" % n][:] *= 0.1
        v["l0.mix.q.b"][0::dim] = 1.0                    # every query has 1 in its first channel ...
        v["l0.mix.k"][0::dim, 0] = gain / 8.0            # ... and token 5's normed input (8 in channel 0) answers with `gain`
        v["l0.mix.r1"][:] = r
        v["l0.mix.sink"][:] = -3.0 if sink is None else sink
    return Model(cfg, seed=11, edit=edit)


@BOTH
@pytest.mark.parametrize("dim,vdim", [(48, 32), (128, 96)])
@pytest.mark.parametrize("window", [2, 16, 63, 64, 65, 128, 130])
def test_window_edge_in_prompts_and_decoding(window, dim, vdim, f32):
    m = standout(window, dim=dim, vdim=vdim)
    n = 2 * window + 80
    for place in (0, 7, 63, 64):
        t = [(3 + i) % 5 for i in range(n)]
        t[place] = 5
        want = m.ref(t)
        inside, outside = place + window - 1, place + window
        moved = err(want[outside], want[inside])
        assert moved > 0.2, "the input does not show the edge: %g" % moved
        got = m.dec(f32, max_seq=512).prefill_logits(t)
        d = m.dec(f32, max_seq=512)
        cut = max(1, inside - 2)
        d.prefill_logits(t[:cut], want=[])
        dec = decode(d, t[cut:outside + 3], cut)
        tol = 1e-4 if f32 else 3e-2
        for p in (place, place + 1, inside - 1, inside, outside, outside + 1, n - 1):
            if p < n:
                assert err(got[p], want[p]) < tol, (window, place, p)
            if cut <= p < outside + 3:
                assert err(dec[p - cut], want[p]) < tol, (window, place, p)


@BOTH
def test_far_key_behind_hundreds_of_others(f32):
    """One key far back holds half the weight; a distance bias that is off by one place or a lost row would show."""
    m = standout(1000, r=0.3, gain=9.0)
    t = [(3 + i) % 5 for i in range(700)]
    t[2] = 5
    want = m.ref(t)
    d = m.dec(f32, max_seq=1024)
    got = d.prefill_logits(t[:640])
    rows = [3, 63, 64, 65, 127, 128, 300, 511, 512, 513, 639]
    assert err(got[rows], want[rows]) < (1e-4 if f32 else 3e-2)
    assert err(decode(d, t[640:], 640), want[640:]) < (1e-4 if f32 else 3e-2)


@BOTH
@pytest.mark.parametrize("sink", [-20.0, 2.0, 5.0])
def test_sink(sink, f32):
    m = standout(30, sink=sink, gain=2.0)
    t = [5] + [(3 + i) % 5 for i in range(70)]
    want = m.ref(t)
    d = m.dec(f32)
    assert err(d.prefill_logits(t[:66]), want[:66]) < (1e-4 if f32 else 3e-2)
    assert err(decode(d, t[66:], 66), want[66:]) < (1e-4 if f32 else 3e-2)
    other = standout(30, sink=sink + 1.0, gain=2.0).ref(t)
    assert sink < -10 or err(other, want) > 0.03


@BOTH
@pytest.mark.parametrize("kind", ["retention", "general_delta"])
def test_state_remembers_a_far_token(kind, f32):
    """Slow decay and one large token: what it left in the state still moves the logits hundreds of tokens later."""
    lay = retention(heads=2, dim=16, vdim=16, dims=8, decay=[0.9995, 0.999]) if kind == "retention" else delta(heads=2, dim=16)
    cfg = config([lay], width=64, ff=0, vocab=40)

    def edit(v):
        if kind == "general_delta":
            v["l0.mix.w0"][:] = -9.0               # hardly any decay
            v["l0.mix.w2"][:] = 0.0
            v["l0.mix.a.b"][:] = -7.0              # hardly any removal
    m = Model(cfg, seed=12, edit=edit)
    t = [7] + [(3 + i) % 6 for i in range(600)]
    other = [8] + t[1:]
    want = m.ref(t)
    assert err(m.ref(other)[600], want[600]) > 1e-3
    d = m.dec(f32, max_seq=700)
    got = run_portions(d, t[:560], [100, 2, 33])
    assert err(got, want[:560]) < TOL[f32]
    assert err(decode(d, t[560:], 560), want[560:]) < TOL[f32]


@BOTH
def test_long_decoding(f32):
    m = Model(config([retention(), attention(window=50), delta()]), seed=13)
    t = toks(400)
    assert err(decode(m.dec(f32, max_seq=400), t, 0), m.ref(t)) < TOL[f32]


@BOTH
def test_prompt_longer_than_a_chunk(f32):
    """2,100 tokens: the session cuts a prompt after 2,048."""
    m = Model(config([attention(heads=2, kv=1, dim=80, vdim=80, window=300), retention(heads=1, dim=16, vdim=16), delta(heads=1, dim=16)], width=32, ff=0), seed=14)
    t = toks(2100)
    want = m.ref(t)
    rows = [0, 1, 2046, 2047, 2048, 2049, 2099]
    got = m.dec(f32, max_seq=2200).prefill_logits(t, want=rows)
    assert err(got, want[rows]) < TOL[f32]
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
        lg = tl.Tensor.from_numpy(d2.logits())
        tok = lg.sample_top_k_top_p(0.8, 20, 0.9, tl.rng_uniform(4, i)).item_i64()
        assert tok == got[i], i


def test_model_folder_loads_to_the_same_model(tmp_path):
    m = Model(config(MIXED), seed=17)
    synth.write_model_dir(tmp_path / "m", m.cfg, m.bits)
    w = tl.TensorMap.load_dir(tmp_path / "m")
    assert w.meta_string("general.architecture") == "Mukutar" and w.decoder_cfg()["n_layers"] == len(MIXED)
    t = toks(50)
    a = tl.Decoder(None, w, max_seq=64, f32=True).prefill_logits(t)
    assert np.array_equal(a, m.dec(True, max_seq=64).prefill_logits(t))
    assert np.array_equal(w.get("l0.norm1").numpy(), synth.from_bf16(m.bits["l0.norm1"]))


def test_missing_or_misshapen_tensors_are_refused():
    cfg = config(MIXED)
    for change, code in ((lambda b: b.pop("l1.mix.sink"), 8), (lambda b: b.pop("l0.mix.g"), 8), (lambda b: b.update({"l2.mix.w2": b["l2.mix.w2"][:-1]}), 1),
                         (lambda b: b.update({"final.norm": b["final.norm"][:-1]}), 1)):
        bits = synth.mukutar_tensors(cfg, 1, 11)
        change(bits)
        w = tl.TensorMap.new()
        for n, b in bits.items():
            w.add(n, synth.BF16, b.shape, np.ascontiguousarray(b))
        w.set_config(json.dumps(cfg))
        with pytest.raises(tl.TlbError) as e:
            tl.Decoder(None, w, max_seq=32)
        assert e.value.code == code
    with pytest.raises(tl.TlbError):
        tl.Decoder(None, Model(cfg).map, max_seq=32, tp_size=2)


def test_prefill_logits_of_a_llama_session(orc):
    """The entry point for logits of several tokens serves the Llama chain too."""
    cfg = dict(n_layers=2, d_model=256, n_heads=4, n_kv_heads=2, head_dim=64, ffn=512, vocab=320, eps=1e-5, rope_base=10000.0, attn_scale=0.125)
    w = tl.map_from_tensors(synth.llama_tensors(cfg, 3, synth.Q4_K, synth.Q6_K))
    t = toks(40, 320)
    d = tl.Decoder(cfg, w, kv_f16=True, max_seq=64)
    got = d.prefill_logits(t, want=[39, 7, 20])
    for row, n in zip(got, (40, 8, 21)):
        d2 = tl.Decoder(cfg, w, kv_f16=True, max_seq=64)
        d2.prefill(t[:n])
        assert np.max(np.abs(row - d2.logits())) < 2e-2 * np.max(np.abs(row))


def test_command_line_generates_from_a_folder_and_from_gguf(tmp_path, capsys):
    from tl_b200 import generate
    m = Model(config(MIXED), seed=15)
    synth.write_model_dir(tmp_path / "m", m.cfg, m.bits)
    prompt = toks(45, seed=5)
    args = ["--model", str(tmp_path / "m"), "--tokens", ",".join(map(str, prompt)), "--f32"]
    generate.main(args + ["-n", "12"])
    assert [int(x) for x in capsys.readouterr().out.split(",")] == greedy(m, prompt, 12)[0]
    generate.main(args + ["-n", "9", "--temp", "0.9", "--top-k", "30", "--seed", "3"])
    a = capsys.readouterr().out
    generate.main(args + ["-n", "9", "--temp", "0.9", "--top-k", "30", "--seed", "3"])
    assert a == capsys.readouterr().out and len(a.split(",")) == 9
    cfg = dict(n_layers=1, d_model=256, n_heads=4, n_kv_heads=2, head_dim=64, ffn=512, vocab=320)
    tens = synth.llama_tensors(dict(cfg, eps=1e-5, rope_base=1e4, attn_scale=0.125), 3, synth.Q4_K, synth.Q6_K)
    meta = {"general.architecture": "llama", "llama.block_count": 1, "llama.embedding_length": 256, "llama.attention.head_count": 4,
            "llama.attention.head_count_kv": 2, "llama.feed_forward_length": 512}
    synth.write_gguf(tmp_path / "l.gguf", tens, metadata=meta)
    generate.main(["--model", str(tmp_path / "l.gguf"), "--tokens", "1,2,3,4,5,6", "-n", "5"])
    assert len(capsys.readouterr().out.split(",")) == 5


def test_trace_replay(tmp_path):
    """bin/trace_run: the logits of the wanted tokens, whatever the portions, for requests one after the other."""
    import os
    import subprocess
    import sys
    m = Model(config(MIXED), seed=18)
    synth.write_model_dir(tmp_path / "m", m.cfg, m.bits)
    a, b = toks(30, seed=1), toks(9, seed=2)
    wa, wb = m.ref(a), m.ref(b)
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
                assert err(np.frombuffer(f.read_bytes(), dtype="<f4").reshape(-1, m.cfg["vocab"]), w) < TOL[dtype == "float32"]
