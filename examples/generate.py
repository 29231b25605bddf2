"""Generate text from a checkpoint: HF-style ``generate()`` (greedy, sampling, beam search) or the CUDA-graph
greedy decoder, optionally tensor-parallel or through the deployment launcher.

    python examples/generate.py --model gptj --checkpoint out/merged --prompt "Hello" --max-new-tokens 64
    python -m torch.distributed.run --nproc-per-node 4 --master-addr 127.0.0.1 examples/generate.py \
        --model gptj --checkpoint out --tp 4 --num-beams 5 --no-repeat-ngram-size 2
    python examples/generate.py --model gptj --checkpoint out/merged --tp 4 --deployment    # one parent, 4 GPU workers
    python examples/generate.py --model auto --checkpoint moronex --dtype bfloat16 --cuda-graph  # family from config.json

Mirrors the reference's ``tests/*/ *_test_kernel_fusion.py`` / ``*_test_deployment.py`` usage. Prompts are encoded
as UTF-8 bytes unless ``--tokenizer`` names a Hugging Face tokenizer directory.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
import time

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))

import oslo_b200 as ob  # noqa: E402

CLASSES = {name: entry.causal_lm for name, entry in ob.MODELS.items()}


def main() -> None:
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", default="gptj", choices=sorted(CLASSES) + ["auto"],
                    help="auto: the family the checkpoint's config.json names")
    ap.add_argument("--checkpoint", required=True)
    ap.add_argument("--dtype", choices=["float32", "bfloat16", "float16"], help="parameter dtype (default: float32)")
    ap.add_argument("--tp", type=int, default=1)
    ap.add_argument("--deployment", action="store_true")
    ap.add_argument("--prompt", nargs="+", default=["Hello"], help="one or more prompts; several run as one left-padded batch")
    ap.add_argument("--tokenizer")
    ap.add_argument("--max-new-tokens", type=int, default=32)
    ap.add_argument("--num-beams", type=int, default=1)
    ap.add_argument("--do-sample", action="store_true")
    ap.add_argument("--top-k", type=int, default=None)
    ap.add_argument("--top-p", type=float, default=None)
    ap.add_argument("--temperature", type=float, default=None)
    ap.add_argument("--no-repeat-ngram-size", type=int, default=None)
    ap.add_argument("--cuda-graph", action="store_true", help="greedy decoding as one CUDA-graph replay per token")
    args = ap.parse_args()

    if args.tokenizer:
        from transformers import AutoTokenizer
        tok = AutoTokenizer.from_pretrained(args.tokenizer)
        encode, decode = (lambda s: tok.encode(s)), (lambda ids: tok.decode(ids))
    else:
        encode = lambda s: list(s.encode("utf-8"))                                            # noqa: E731
        decode = lambda ids: bytes(int(i) for i in ids if 0 <= int(i) < 256).decode("utf-8", "replace")  # noqa: E731

    on_gpu = torch.cuda.is_available() and os.environ.get("OSLO_B200_BACKEND", "nccl") != "gloo"
    if args.model == "auto":
        with open(os.path.join(args.checkpoint, "config.json"), encoding="utf-8") as f:
            cls = ob.find_model(json.load(f)).causal_lm
    else:
        cls = CLASSES[args.model]
    dtype = {"torch_dtype": getattr(torch, args.dtype)} if args.dtype else {}
    if args.tp > 1 or args.deployment:
        model = cls.from_pretrained_with_parallel(args.checkpoint, tensor_parallel_size=args.tp,
                                                  deployment=args.deployment or None, **dtype)
        device = torch.device("cpu") if args.deployment else model.mpu.device
    else:
        model = cls.from_pretrained(args.checkpoint, **dtype)
        device = torch.device("cuda") if on_gpu else torch.device("cpu")
        model = model.to(device)
    if on_gpu and not args.deployment:
        model.fuse()
    model.eval()
    rows = [encode(p) for p in args.prompt]
    longest = max(len(r) for r in rows)
    ids = torch.tensor([[0] * (longest - len(r)) + r for r in rows], dtype=torch.long, device=device)
    kw = dict(max_new_tokens=args.max_new_tokens, num_beams=args.num_beams, do_sample=args.do_sample,
              top_k=args.top_k, top_p=args.top_p, temperature=args.temperature,
              no_repeat_ngram_size=args.no_repeat_ngram_size)
    if any(len(r) != longest for r in rows):
        kw["attention_mask"] = torch.tensor([[0] * (longest - len(r)) + [1] * len(r) for r in rows], device=device)
    if args.cuda_graph:
        kw["cuda_graph"] = True
    if on_gpu and args.no_repeat_ngram_size:
        kw["fused_no_repeat_ngram_blocking"] = True
    t0 = time.perf_counter()
    out = model.generate(ids, **{k: v for k, v in kw.items() if v is not None})
    dt = time.perf_counter() - t0
    if int(os.environ.get("RANK", "0")) == 0:
        for i in range(out.size(0)):
            r = i * len(rows) // out.size(0)
            print(decode(out[i, longest - len(rows[r]):].tolist()))
        print(f"[{out.size(1) - longest} new tokens in {dt:.2f} s]", file=sys.stderr)


if __name__ == "__main__":
    main()
