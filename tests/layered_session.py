"""What the GPU tests of the layered designs share: a model in the library and in plain numpy, sessions fed in portions, errors."""
import json

import numpy as np

import tl_b200 as tl
from tl_b200 import synth


class Model:
    """cfg with tensors of `specs` (name -> shape) valued by `value(name, shape, seed)`, edited before they are rounded to bf16."""

    def __init__(self, cfg, specs, value, plain, seed=1, edit=None):
        self.cfg = cfg
        vals = {n: value(n, s, seed) for n, s in specs.items()}
        if edit:
            edit(vals)
        self.bits = {n: synth.to_bf16(v) for n, v in vals.items()}
        self.plain = plain(cfg, {n: synth.from_bf16(b) for n, b in self.bits.items()})
        self.map = tl.TensorMap.new()
        for n, b in self.bits.items():
            self.map.add(n, synth.BF16, b.shape, b)
        self.map.set_config(json.dumps(cfg))

    def dec(self, f32, max_seq=256, **kw):
        return tl.Decoder(None, self.map, max_seq=max_seq, f32=f32, **kw)

    def ref(self, tokens):
        return self.plain.forward(tokens, self.plain.new_state())


def toks(n, vocab=131, seed=0):
    return [int(t) for t in np.random.default_rng(seed).integers(0, vocab, n)]


def row_errors(a, b):
    """Root mean square over the vocabulary of every row, relative to the logits' own."""
    a, b = np.atleast_2d(a), np.atleast_2d(b)
    d = a - b
    return np.sqrt(np.mean(d * d, axis=1)) / np.sqrt(np.mean(b * b))


def err(a, b):
    return float(np.max(row_errors(a, b)))


def decode(d, tokens, pos):
    out = []
    for i, t in enumerate(tokens):
        d.step(t, pos + i, read=False)
        out.append(d.logits())
    return np.stack(out)


def run_portions(d, tokens, sizes, seq=0, at=0):
    """The tokens from place `at` on, in portions of the given sizes in turn."""
    out, i = [], 0
    while at < len(tokens):
        n = min(sizes[i % len(sizes)], len(tokens) - at)
        out.append(d.prefill_logits(tokens[at:at + n], at, seq=seq))
        at, i = at + n, i + 1
    return np.concatenate(out)


def greedy(m, prompt, n):
    """n greedy tokens behind the prompt by the plain statement, and the smallest gap between the best two logits."""
    st = m.plain.new_state()
    lg = m.plain.forward(prompt, st)[-1]
    out, gaps = [], []
    for _ in range(n):
        top = np.sort(lg)[-2:]
        gaps.append(top[1] - top[0])
        out.append(int(np.argmax(lg)))
        lg = m.plain.forward([out[-1]], st)[-1]
    return out, min(gaps) / np.sqrt(np.mean(lg * lg))
