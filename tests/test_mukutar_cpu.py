"""Host side of the models described by a config.json: registry, config checks, safetensors reader, and the plain statement of the
mechanisms against closed forms.  No device is needed."""
import copy
import ctypes as C
import json
import struct

import numpy as np
import pytest

import plain_layers as P
from tl_b200 import _lib, synth

CFG = {"architecture": "Mukutar", "vocab": 61, "width": 40, "norm": {"eps": 1e-5}, "layers": [
    {"type": "attention", "mixer": {"heads": 6, "kv_heads": 3, "dim": 10, "vdim": 14, "scale": 0.3, "mask": {"size": 9}}, "mlp": {"kind": "dense", "ff": 52}},
    {"type": "retention", "mixer": {"heads": 2, "dim": 12, "vdim": 20, "rot": {"base": 500.0, "dims": 8}, "decay": [0.9, 0.99]}, "mlp": None},
    {"type": "general_delta", "mixer": {"heads": 3, "dim": 11}, "mlp": {"kind": "dense", "ff": 30}}]}


def set_config(cfg):
    m = C.c_void_p()
    L = _lib.lib()
    assert L.tlb_map_new(C.byref(m)) == 0
    st = L.tlb_map_set_config(m, (cfg if isinstance(cfg, str) else json.dumps(cfg)).encode())
    arch = L.tlb_map_meta_string(m, b"general.architecture")
    dc = _lib.DecoderCfg()
    sizes = (dc.n_layers, dc.d_model, dc.vocab) if st else None
    if st == 0:
        assert L.tlb_decoder_cfg_from_map(m, C.byref(dc)) == 0
        sizes = (dc.n_layers, dc.d_model, dc.vocab)
    L.tlb_map_free(m)
    return st, arch, sizes


def test_registry_reads_a_config():
    st, arch, sizes = set_config(CFG)
    assert st == 0 and arch == b"Mukutar" and sizes == (3, 40, 61)


@pytest.mark.parametrize("change,status", [
    (lambda c: c.update(architecture="Nope"), 7), (lambda c: c.pop("architecture"), 8), (lambda c: c.pop("vocab"), 8),
    (lambda c: c.update(width=0), 8), (lambda c: c.update(width=2.5), 8), (lambda c: c.update(layers=[]), 8), (lambda c: c.pop("norm"), 8),
    (lambda c: c["layers"][0].update(type="mamba"), 7), (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), 8),
    (lambda c: c["layers"][0]["mixer"].pop("mask"), 8), (lambda c: c["layers"][0]["mixer"].pop("scale"), 8),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5]), 8), (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), 8),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=14), 8), (lambda c: c["layers"][2].update(mlp={"kind": "moe", "ff": 8}), 7),
    (lambda c: c["layers"][2]["mlp"].pop("ff"), 8), (lambda c: c["layers"].append(5), 8)])
def test_registry_refuses_what_it_cannot_run(change, status):
    c = copy.deepcopy(CFG)
    change(c)
    assert set_config(c)[0] == status


def test_registry_refuses_text_that_is_no_object():
    for text in ("", "[1, 2]", "{\"architecture\": ", "null"):
        assert set_config(text)[0] == 8


def load_dir(path):
    m = C.c_void_p()
    st = _lib.lib().tlb_model_load(C.byref(m), str(path).encode())
    if st == 0:
        _lib.lib().tlb_map_free(m)
    return st


def test_hostile_model_folders_are_clean_errors(tmp_path):
    """Lengths and offsets of an untrusted safetensors file neither wrap the bounds checks nor reach an allocation."""
    assert load_dir(tmp_path / "none") == 8
    d = tmp_path / "m"
    d.mkdir()
    (d / "config.json").write_text(json.dumps(CFG))
    assert load_dir(d) == 8                                                       # no model.safetensors
    f = d / "model.safetensors"
    entry = lambda **kw: json.dumps({"embed": dict({"dtype": "BF16", "shape": [2, 2], "data_offsets": [0, 8]}, **kw)}).encode()
    blob = lambda head, data=b"\0" * 8, n=None: struct.pack("<Q", len(head) if n is None else n) + head + data
    for raw in (b"", b"\1\0\0", blob(b"{}", n=1 << 62), blob(b"{}", n=0xFFFFFFFFFFFFFFF8), blob(b"[1]"), blob(b"{\"a\": "), blob(b"{\"a\": 3}"),
                blob(entry(data_offsets=[0, 16])), blob(entry(data_offsets=[8, 0])), blob(entry(data_offsets=[0])), blob(entry(data_offsets=[-8, 0])),
                blob(entry(data_offsets=[0, 1e30])), blob(entry(shape=[1.5, 2])), blob(entry(shape=[-2, -2])), blob(entry(shape=[1 << 40, 1 << 40])),
                blob(entry(shape=[1] * 40)), blob(entry(shape="x"))):
        f.write_bytes(raw)
        assert load_dir(d) in (1, 8), raw
    f.write_bytes(blob(entry(dtype="F8_E4M3")))
    assert load_dir(d) == 7


def test_bf16_rounding_and_folder_writer(tmp_path):
    x = np.array([1.0, 1.00390625, 1.01171875, -3.1415927, 1e-30, 0.0], dtype=np.float32)
    back = synth.from_bf16(synth.to_bf16(x))
    assert back[0] == 1.0 and back[1] == 1.0 and back[2] == np.float32(1.015625)       # ties to even, both ways
    assert np.all(np.abs(back - x) <= np.abs(x) * 2.0 ** -8)
    synth.write_model_dir(tmp_path / "w", CFG, {"a": synth.to_bf16(np.ones((3, 2), dtype=np.float32)), "t": np.arange(4, dtype=np.int32)})
    raw = (tmp_path / "w" / "model.safetensors").read_bytes()
    n = struct.unpack("<Q", raw[:8])[0]
    head = json.loads(raw[8:8 + n])
    assert head["a"] == {"dtype": "BF16", "shape": [3, 2], "data_offsets": [0, 12]} and head["t"]["dtype"] == "I32"
    assert np.array_equal(np.frombuffer(raw[8 + n + 12:], dtype=np.int32), np.arange(4))


# ---- the plain statement against closed forms
def test_plain_retention_is_a_decayed_sum():
    r = np.random.default_rng(0)
    q, k, v = r.standard_normal((3, 7, 2, 5))
    dec = np.array([0.7, 0.95])
    S, outs = np.zeros((2, 5, 5)), []
    for t in range(7):
        S, o = P.retention_token(S, q[t], k[t], v[t], dec)
        outs.append(o)
    for h in range(2):
        want = sum(dec[h] ** (6 - s) * (q[6, h] @ k[s, h]) * v[s, h] for s in range(7))
        assert np.allclose(outs[6][h], want)


def test_plain_delta_rule_replaces_and_decays():
    """Full removal (a = 1) without decay leaves exactly the new value along the key; zero removal only decays."""
    r = np.random.default_rng(1)
    S = r.standard_normal((1, 6, 6))
    k = r.standard_normal((1, 6))
    v = r.standard_normal((1, 6))
    one, zero = np.ones((1, 6)), np.zeros((1, 6))
    S2, _ = P.general_delta_token(S, zero, k, v, one, one)
    u = k[0] / np.linalg.norm(k[0])
    assert np.allclose(u @ S2[0], np.linalg.norm(k[0]) * v[0], atol=1e-5)
    w = r.uniform(0.6, 1.0, (1, 6))
    S3, o = P.general_delta_token(S, one, zero, v, w, zero)
    assert np.allclose(S3[0], w[0][:, None] * S[0]) and np.allclose(o[0], S3[0].sum(0))


def test_plain_attention_window_sink_and_bias():
    r = np.random.default_rng(2)
    ks, vs, q = r.standard_normal((6, 1, 4)), r.standard_normal((6, 1, 3)), r.standard_normal((2, 4))
    z = np.zeros(2)
    out = P.attention_token(q, ks, vs, 0.5, z, z, np.full(2, -1e9), 1)
    assert np.allclose(out, vs[5])                                                  # itself only
    out = P.attention_token(q, ks, vs, 0.0, z, z, np.log(3.0) * np.ones(2), 3)
    assert np.allclose(out[0], vs[3:, 0].sum(0) / 6.0)                              # three equal scores and a sink worth three
    out = P.attention_token(q, ks, vs, 0.0, np.ones(2), np.ones(2), np.full(2, -1e9), 2)
    assert np.allclose(out[0], (vs[5, 0] + vs[4, 0] / 2) / 1.5)                     # exp(-ln 2) for the neighbour


def test_plain_rotation_turns_pairs_by_their_angle():
    x = np.arange(12.0).reshape(1, 12)
    y = P.rotate_half(x, 3, 100.0, 8)
    assert np.array_equal(y[0, 8:], x[0, 8:])
    for i in range(4):
        z = complex(x[0, i], x[0, i + 4]) * np.exp(1j * 3 * 100.0 ** (-2 * i / 8))
        assert np.allclose([y[0, i], y[0, i + 4]], [z.real, z.imag])


def test_plain_poly_norm_has_unit_terms():
    z = np.random.default_rng(3).standard_normal(50)
    for n, c in ((1, (1, 0, 0, 0)), (2, (0, 1, 0, 0)), (3, (0, 0, 1, 0))):
        y = P.poly_norm(z, c, 0.0)
        assert np.isclose(np.mean(y * y), 1.0) and np.allclose(y / y[0], (z / z[0]) ** n)
    assert np.allclose(P.poly_norm(z, (0, 0, 0, 0.25), 1e-5), 0.25)
