"""Small Sinorax models and the ways of running them that the CPU and the GPU tests share.

The configurations differ from each other in every size and option: layer orders, groups of 1 to 4 query heads, keys and values of
different sizes, heads turned in part and in full, with and without a factor on the frequencies, windows of one position, shorter and
longer than a page, none; layers without feed-forward; a bigram table of one bucket, of many, with multipliers whose products pass 32
bits, or none; logits with and without factor and bound. The engine runs them through ``TraceReplayer`` (the step function, the
cache manager, the kernels object it is given); the oracle is ``plain_sinorax.forward`` on whole sequences.
"""
from __future__ import annotations

import json
from pathlib import Path

import torch

import plain_sinorax as plain
from luvutar_cases import cuts_of, load_plain, prompt, row_error, run_alone, run_mixed  # noqa: F401  (generic helpers)


def _turned(heads, kv_heads, dim, vdim, scale, dims, base, factor=None, ff=None):
    rot = {"dims": dims, "base": base}
    if factor:
        rot["scaling"] = {"factor": factor}
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def _sigmoid(heads, kv_heads, dim, vdim, scale, window, ff=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        m["mask"] = {"size": window}
    return {"type": "attention_2", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def _model(vocab, width, layers, bigram=None, scale=None, cap=None):
    d = {"architecture": "Sinorax", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "layers": layers}
    if bigram:
        d["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}
    if scale:
        d["logit_scale"] = scale
    if cap:
        d["logit_softcap"] = cap
    return d


CASES = {
    # (config, page size). A: partly turned heads, values shorter and longer than keys, windows longer and shorter than a page of 8, a
    # sigmoid layer first, a layer without feed-forward
    "A": (_model(83, 48, [_sigmoid(6, 3, 16, 24, 0.25, 19, ff=56), _turned(4, 2, 24, 16, 0.2, 16, 900.0, 2.5, ff=40),
                          _sigmoid(2, 1, 32, 32, 0.3, 5), _turned(3, 3, 16, 40, 0.3, 8, 50.0, ff=64)], (61, 13, 5), 0.7, 20.0), 8),
    # B: sizes that the tensor-core kernels take: heads of 64, 96 and 128, fully turned and half, groups of 4, 1 and 2
    "B": (_model(120, 64, [_turned(8, 2, 64, 64, 0.125, 64, 10000.0, ff=96), _sigmoid(4, 1, 64, 128, 0.2, 40, ff=72),
                           _turned(2, 2, 128, 128, 0.1, 64, 300.0, 8.0), _sigmoid(3, 3, 96, 96, 0.1, 130, ff=32),
                           _turned(4, 4, 96, 64, 0.1, 32, 2000.0, 1.5, ff=40), _sigmoid(4, 2, 128, 64, 0.15, 16, ff=48)], (997, 2000000011, 1999999973), 1.5, 12.0), 16),
    # C: sizes that take the kernels' slow paths (a width that is no multiple of 8, heads of 10, 20 and 14, values of 6, 7 and 22), a window of one
    # position, a bigram table of a single bucket, plain frequencies, neither factor nor bound on the logits; pages of 4
    "C": (_model(57, 44, [_turned(3, 1, 10, 6, 0.35, 2, 7.0, ff=52), _sigmoid(5, 5, 20, 7, 0.22, 1, ff=20), _turned(2, 2, 14, 22, 0.3, 14, 40.0, 3.0)],
                 (1, 1, 1)), 4),
    # D: no bigram table; a sigmoid layer that sees every earlier position; two kinds of windowed layers whose pages part ways
    "D": (_model(64, 40, [_sigmoid(4, 4, 16, 16, 0.25, None, ff=48), _sigmoid(4, 2, 16, 16, 0.25, 33, ff=24), _turned(5, 1, 32, 32, 0.2, 32, 500.0, 0.5, ff=36)],
                 None, 2.0), 16),
}

# float32: only the order of summation differs. bfloat16: activations are rounded to 8 bits between the kernels, and every sublayer's
# result is brought back to full size by its closing Dynamic Tanh; a wrong key or a lost token moves the logits by 0.3 and more
LIMIT = {"float32": 3e-5, "bfloat16": 8e-2}
LENS = {"a": 150, "b": 67, "c": 41, "d": 9, "e": 118, "f": 2}


def make_folder(tmp: Path, name: str, store: str = "float32", std: float = 0.08, seed: int = 11, sharp: float = 1.0) -> Path:
    """A model folder for case ``name`` with random weights whose mechanisms all show: slopes between 0.3 and 1.2, large biases and
    bigram rows, sigmoid offsets of both signs. ``sharp`` multiplies the query projections, so that few keys matter and one that is
    lost, or seen when it should not be, moves the logits by far more than rounding does."""
    from llm_infrence_engine_b200.weights.random_init import random_tensors
    from llm_infrence_engine_b200.weights.safetensors_io import write_safetensors

    cfg, _ = CASES[name]
    t = random_tensors(cfg, seed, std)
    g = torch.Generator().manual_seed(seed + 1)
    for key in t:
        if key.endswith(".alpha"):
            t[key] = 0.3 + 0.9 * torch.rand((), generator=g)
        elif key.endswith(".pb"):
            t[key] = torch.randn(t[key].shape, generator=g) - 1.0
        elif key in ("embed", "bigram"):
            t[key] = torch.randn(t[key].shape, generator=g) * 0.7
        elif ".mix." in key and key.endswith(".b"):
            t[key] = torch.randn(t[key].shape, generator=g) * 0.4
        elif key == "head":
            t[key] = torch.randn(t[key].shape, generator=g) * 0.2
        if sharp != 1.0 and key.endswith("mix.q"):
            t[key] = t[key] * sharp
    dtype = {"float32": torch.float32, "bfloat16": torch.bfloat16}[store]
    folder = Path(tmp) / f"sinorax_{name}_{store}_{sharp}"
    folder.mkdir(parents=True, exist_ok=True)
    write_safetensors(folder / "model.safetensors", {k: v.to(dtype).contiguous() for k, v in t.items()})
    (folder / "config.json").write_text(json.dumps(cfg))
    return folder


def replayer(folder, name, dtype, max_tokens, kernels=None, device="cuda:0", **kw):
    from llm_infrence_engine_b200.engine import TraceReplayer

    return TraceReplayer(str(folder), dtype, max_tokens, device=device, kernels=kernels, block_size=CASES[name][1], **kw)


def plain_logits(cfg, tensors, tokens):
    return plain.forward(cfg, tensors, tokens, torch.float64)


def setup_case(tmp, name, dtype, **kw):
    folder = make_folder(tmp, name, dtype, **kw)
    cfg, tensors = load_plain(folder)
    prompts = {k: prompt(cfg["vocab"], n, 3 + i) for i, (k, n) in enumerate(LENS.items())}
    want = {k: plain_logits(cfg, tensors, p) for k, p in prompts.items()}
    return folder, cfg, tensors, prompts, want


# ---------------------------------------------------------------------------------------------------------------------
# The checks themselves: each takes the kernels object and the device, so the same statements run on the CPU (torch
# stand-in kernels: the host side of the engine) and on the GPU (the package's kernels).

def check_whole_and_cut(case, name, dtype, kernels, device, only=None):
    """Whole prompts; the last tokens one by one; portions of several sizes down to two tokens and one."""
    folder, cfg, tensors, prompts, want = case
    rp = replayer(folder, name, dtype, 192, kernels, device)
    n = 0
    for k, p in prompts.items():
        if only and k not in only:
            continue
        T = len(p)
        ways = {"whole": [(0, T)], "tail one by one": cuts_of(T, [max(1, T - 40)] + [1] * 40),
                "portions": cuts_of(T, [7, 2, 33, 1, 16, 3, 2, 64, 5]), "pairs": cuts_of(T, [2])}
        for what, cuts in ways.items():
            if what == "pairs" and T > 70:
                continue
            got = run_alone(rp, f"{k}{n}", p, cuts, n)
            n += len(cuts)
            err = row_error(got, want[k])
            assert err <= LIMIT[dtype], f"{name} {dtype} request {k} ({T} tokens) {what}: {err:.3g}"
            rp.cache.check_invariants()
    assert rp.cache.num_free_slots() == 4 and all(p.num_free == p.capacity for p in rp.cache.pools)


def check_mixed(case, name, dtype, kernels, device, seeds=(0, 1)):
    """Batches of unequal requests on a pool that holds only the live ones (pages and state slots are used again): every
    request as if it ran alone."""
    folder, cfg, tensors, prompts, want = case
    for seed in seeds:
        lens = sorted((len(p) for p in prompts.values()), reverse=True)
        rp = replayer(folder, name, dtype, sum(-(-n // 64) * 64 for n in lens[:4]), kernels, device)
        got = run_mixed(rp, prompts, seed)
        for k in prompts:
            err = row_error(got[k], want[k])
            assert err <= LIMIT[dtype], f"{name} {dtype} mixed (seed {seed}) request {k}: {err:.3g}"
        assert rp.cache.num_free_slots() == 4 and all(p.num_free == p.capacity for p in rp.cache.pools)


def check_long_decoding(case, name, dtype, kernels, device, total=300):
    """A short prompt, then hundreds of tokens one by one: windows pass over decoded tokens and give their pages back."""
    folder, cfg, tensors, prompts, want = case
    p = prompt(cfg["vocab"], total, 99)
    ref = plain_logits(cfg, tensors, p)
    rp = replayer(folder, name, dtype, 320, kernels, device)
    got = run_alone(rp, "long", p, cuts_of(total, [3] + [1] * total))
    err = row_error(got, ref)
    assert err <= LIMIT[dtype], f"{name} {dtype} long decoding: {err:.3g}"
    first = row_error(got[:4], ref[:4])
    assert first <= LIMIT[dtype], f"{name} {dtype} first tokens: {first:.3g}"


def check_slot_reuse(case, name, dtype, kernels, device):
    """One request after another on the same slot, each beginning with a single token: the first token of a request takes the
    bigram table's last row whatever the slot's earlier owner left there, the second one the first token's row."""
    folder, cfg, tensors, prompts, want = case
    rp = replayer(folder, name, dtype, 192, kernels, device)
    for n, (k, p) in enumerate(prompts.items()):
        p, ref = p[:12], want[k][:12]
        got = run_alone(rp, f"s{n}", p, cuts_of(len(p), [1, 1, 2, 1, 3, 4]), 100 * n)
        err = row_error(got, ref)
        assert err <= LIMIT[dtype], f"{name} {dtype} request {k} on a used slot: {err:.3g}"
