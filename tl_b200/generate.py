"""Generation from the command line, for every model the library loads: a GGUF file of a Llama model, or a model folder
(config.json + model.safetensors).

    python -m tl_b200.generate --model PATH --tokens 1,15,7 [-n 32] [--temp T --top-k K --top-p P --seed S] [--f32]
    python -m tl_b200.generate --model PATH --tokenizer tokenizer.json --prompt "..." [...]

Prints the generated ids, and their text when a tokenizer is given.  temp 0 (the default) is greedy.
"""
import argparse
import os


def load(path):
    """(config or None, tensor map) of a GGUF file or a model folder."""
    from . import TensorMap
    if os.path.isdir(path):
        return None, TensorMap.load_dir(path)
    m = TensorMap.load(path)
    return m.decoder_cfg(), m


def generate(path, tokens, n, temp=0.0, top_k=0, top_p=1.0, seed=0, f32=False, max_seq=None):
    """n tokens behind `tokens`: the prompt in one pass, then the session's decode loop on the device."""
    from . import Decoder, Tensor, rng_uniform
    cfg, weights = load(path)
    dec = Decoder(cfg, weights, max_seq=max_seq or len(tokens) + n + 1, f32=f32)
    first = dec.prefill(tokens)
    if n < 1:
        return []
    if temp > 0:
        # the first token by the same sampler; the session draws the following ones from counters 0, 1, ... of the seed
        first = Tensor.from_numpy(dec.logits()).sample_top_k_top_p(temp, top_k, top_p, rng_uniform(seed, (1 << 64) - 1)).item_i64()
        return [first] + dec.generate_sampled(first, len(tokens), n - 1, temp, top_k, top_p, seed)
    return [first] + dec.generate(first, len(tokens), n - 1)


def main(argv=None):
    ap = argparse.ArgumentParser(prog="python -m tl_b200.generate", description="Generate tokens from a GGUF file or a model folder.")
    ap.add_argument("--model", required=True, help="GGUF file, or a folder with config.json and model.safetensors")
    ap.add_argument("--tokens", help="prompt as token ids with commas between them")
    ap.add_argument("--prompt", help="prompt as text (needs --tokenizer)")
    ap.add_argument("--tokenizer", help="tokenizer.json")
    ap.add_argument("-n", type=int, default=32, help="tokens to generate")
    ap.add_argument("--temp", type=float, default=0.0)
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--f32", action="store_true", help="all products in 32 bits (model folders)")
    ap.add_argument("--max-seq", type=int, help="cache rows (default: what the run needs)")
    a = ap.parse_args(argv)
    tok = None
    if a.tokenizer:
        from . import Tokenizer
        tok = Tokenizer(a.tokenizer)
    if a.tokens:
        ids = [int(x) for x in a.tokens.split(",")]
    elif a.prompt is not None and tok:
        ids = tok.encode_ids(a.prompt)
    else:
        ap.error("give --tokens, or --prompt with --tokenizer")
    out = generate(a.model, ids, a.n, a.temp, a.top_k, a.top_p, a.seed, a.f32, a.max_seq)
    print(",".join(str(t) for t in out))
    if tok:
        print(tok.decode_ids(out))


if __name__ == "__main__":
    main()
