"""``brain pakalix|nezalorn|zepesun|povipel <import|infer|serve|trace>``: hybrid decoders (attention and recurrent layers) on the
serving engine.  ``--model`` takes a directory with ``config.json`` and ``model.safetensors`` or a brain
checkpoint; prompts are text with ``--tokenizer`` or token ids with ``--tokens 1,2,3``."""
from __future__ import annotations

import os
import sys
import time
from typing import List

from .args import Args, canon_verb

_USAGE = "usage: brain %s <import|infer|serve|trace> ..."


def run_hybrid(argv: List[str], device: str = "auto", arch: str = "pakalix") -> int:
    verb = canon_verb(argv[0]) if argv else None
    table = {"import": _import, "infer": _generate, "serve": _generate, "trace": _trace}
    fn = table.get(verb)
    if fn is None:
        print(f"{_USAGE % arch}  (got {verb!r})", file=sys.stderr)
        return 2
    return fn(argv[1:], device, arch) or 0


def _import(args, device, arch):
    """Directory -> one brain checkpoint (configuration in its metadata), optionally into the model store."""
    from ..checkpoint import st
    from ..models.config import HybridConfig
    a = Args(args)
    src = a.take_str("--model") or a.positional()
    out = a.take_str("--out")
    dtype = a.str_or("--dtype", "BF16").upper()
    model_id = a.take_str("--id")
    mdir = a.take_str("--models-dir")
    a.finish()
    if not src:
        print(f"usage: brain {arch} import <DIR> [--out F | --id VENDOR/REPO [--models-dir D]] [--dtype F32|BF16]",
              file=sys.stderr)
        return 2
    try:
        model, _, _ = st.load_model(src)
    except Exception as e:  # noqa: BLE001
        print(f"import failed: {e}", file=sys.stderr)
        return 1
    if not isinstance(model.cfg, HybridConfig):
        print(f"import failed: {src} does not hold a hybrid decoder", file=sys.stderr)
        return 1
    if model_id:
        from ..modelref import ModelRef, RefError
        from ..modelstore import Store, default_root
        try:
            ref = ModelRef.parse(model_id).base()
        except RefError as e:
            print(f"--id: {e}", file=sys.stderr)
            return 2
        root = default_root(mdir)
        if not root:
            print("no models directory resolved (set --models-dir, BRAIN_MODELS_DIR, or HOME)", file=sys.stderr)
            return 1
        from ..checkpoint.card import ModelCard
        store = Store(root)
        os.makedirs(store.repo_dir(ref), exist_ok=True)
        tmp = out or os.path.join(store.repo_dir(ref), ".import.safetensors")
        st.save_model(tmp, model, ModelCard(id=str(ref), family="hybrid", param_count=model.cfg.param_count(),
                                            capabilities=["generate"]), dtype)
        tok = os.path.join(src, "tokenizer.json")
        lm = store.install(ref, tmp, tok if os.path.exists(tok) else None)
        if not out:
            os.remove(tmp)
        print(f"ok: installed {ref} -> {lm.weights}")
        return 0
    out = out or f"{arch}.safetensors"
    st.save_model(out, model, dtype=dtype)
    print(f"ok: wrote {out} ({model.cfg.n_layers} layers, width {model.cfg.width}, vocab {model.cfg.vocab})")


def _generate(args, device, arch):
    from ..checkpoint import st
    from ..models.config import HybridConfig
    from ..serve.offline import serve_prompts
    from ..serve.sampling import SampleParams
    from ..train import pick_device
    a = Args(args)
    src = a.take_str("--model") or a.take_str("--weights") or ""
    tokenizer = a.take_str("--tokenizer")
    prompts = a.take_all("--prompt")
    ids = a.take_all("--tokens")
    max_new = a.int_or("--max-new", 32)
    block_size = a.int_or("--block-size", 16)
    max_batch = a.int_or("--max-batch", 0)
    temp, top_k, top_p = a.float_or("--temp", 0.0), a.int_or("--top-k", 0), a.float_or("--top-p", 1.0)
    seed = a.int_or("--seed", 0)
    dtype = a.str_or("--dtype", "bf16")
    a.finish()
    if not src or not (prompts and tokenizer or ids):
        print(f"usage: brain {arch} infer|serve --model DIR|F (--tokenizer T --prompt \"...\" | --tokens 1,2,3)... "
              "[--max-new N --max-batch B --block-size 16 --temp X --top-k K --top-p P --seed S --dtype bf16|fp32]",
              file=sys.stderr)
        return 2
    dev = pick_device(device)
    if dev.type != "cuda":
        print(f"brain {arch}: the hybrid engine needs a CUDA device", file=sys.stderr)
        return 1
    tok, eos = None, None
    batch = [[int(t) for t in s.split(",") if t.strip()] for s in ids]
    if prompts:
        from ..data.tokenizer import load_tokenizer
        tok = load_tokenizer(tokenizer)
        eos = tok.eos_id
        batch = [tok.encode(p) for p in prompts] + batch
    model, _, _ = st.load_model(src)
    if not isinstance(model.cfg, HybridConfig):
        print(f"{src} does not hold a hybrid decoder", file=sys.stderr)
        return 1
    t0 = time.time()
    r = serve_prompts(model.to(dev), batch, max_new, block_size, "bf16", eos, SampleParams(temp, top_k, top_p), seed,
                      max_batch=max_batch or None, dtype=dtype)
    for i, out in enumerate(r["outputs"]):
        text = tok.decode(out) if tok is not None and i < len(prompts) else ",".join(map(str, out))
        print(text if len(batch) == 1 else f"=== prompt {i}\n{text}")
    print(f"served {len(batch)} prompts, {r['tokens']} tokens in {r['secs']:.2f}s ({r['tok_s']:.1f} tok/s aggregate, "
          f"{time.time() - t0:.2f}s with set-up) [{dtype}]", file=sys.stderr)


def _trace(args, device, arch):
    from ..serve.trace_run import main
    return main(args)
