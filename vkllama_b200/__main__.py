"""Command line: generate token ids from a prompt of token ids.

    python -m vkllama_b200 generate --model PATH --prompt 1,2,3 [--tokens N] [--topk K | --topp P] [--seed S]
    python -m vkllama_b200 info

PATH is a GGUF file (Llama-2) or the folder of a registered decoder design. Greedy without --topk / --topp;
with them every token is drawn by the library's samplers (app/llama2_infer.cpp:141-210 is the reference's loop).
"""
import argparse
import sys

import numpy as np

import vkllama_b200 as vk


def generate(model, prompt, n, topk=0, topp=0.0, seed=0):
    """n ids after `prompt`: the device's own greedy loop, or one sampled token per pass."""
    if not topk and not topp:
        return [int(t) for t in model.generate(prompt, n)[0]]
    sampler = vk.TopPSampler(topp, seed) if topp else vk.TopkSampler(topk, seed)
    ids, at, toks = [], 0, list(prompt)
    for _ in range(n):
        logits = model(toks, at)
        at += len(toks)
        if topp or topk > 64:
            ids.append(int(sampler.sample(logits)))
        else:
            ids.append(int(sampler.sample_candidates(*model.topk(min(topk, logits.size)))))
        toks = ids[-1:]
    return ids


def main(argv=None):
    ap = argparse.ArgumentParser(prog="python -m vkllama_b200")
    sub = ap.add_subparsers(dest="cmd", required=True)
    sub.add_parser("info", help="registered architectures and the device")
    g = sub.add_parser("generate", help="generate token ids")
    g.add_argument("--model", required=True)
    g.add_argument("--prompt", required=True, help="token ids, separated by commas")
    g.add_argument("--tokens", type=int, default=32)
    g.add_argument("--maxlen", type=int, default=0)
    g.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16", help="compute type of a decoder design")
    g.add_argument("--topk", type=int, default=0)
    g.add_argument("--topp", type=float, default=0.0)
    g.add_argument("--seed", type=int, default=0)
    g.add_argument("--device", type=int, default=0)
    a = ap.parse_args(argv)
    if a.cmd == "info":
        print("architectures: llama (GGUF), %s (folder)" % ", ".join(vk.architectures()))
        try:
            name, sms, mem = vk.Device(0).info()
            print("device: %s, %d SMs, %.0f GB" % (name, sms, mem / 1e9))
        except vk.VklError as e:
            print("device: %s" % e.message)
        return 0
    prompt = np.array([int(t) for t in a.prompt.split(",")], np.uint32)
    dev = vk.Device(a.device)
    model = vk.load_model(dev, a.model, a.maxlen, vk.FP32 if a.dtype == "float32" else vk.BF16)
    print(" ".join(str(t) for t in generate(model, prompt, a.tokens, a.topk, a.topp, a.seed)))
    model.close()
    dev.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
