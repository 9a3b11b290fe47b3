"""Small Putelix models and the ways of running them that the CPU and the GPU tests share.

The configurations differ from each other in every size and option: groups of 1 to 4 query heads, heads that the tensor-core kernels
take and heads that they do not, chunks of one position, shorter and longer than a page, none; scores with and without a cap;
distance tables of several sizes; decays of 0, 1 and between; memories whose values are longer and shorter than their keys; dense
feed-forwards, experts of which one, some or all are chosen, shared experts of the experts' width, of another, none; layers without
feed-forward; a position table whose length the checkpoint decides. The engine runs them through ``TraceReplayer`` (the step
function, the cache manager, the kernels object it is given); the oracle is ``plain_putelix.forward`` on whole sequences.
"""
from __future__ import annotations

import json
from pathlib import Path

import torch

import plain_putelix as plain
from luvutar_cases import cuts_of, load_plain, mixed_schedule, prompt, row_error, run_alone  # noqa: F401  (generic helpers)


def _layer(left, right, mlp=None):
    heads, kv_heads, dim, scale, cap, chunk, far = left
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "bias_max": far}
    if cap:
        m["softcap"] = cap
    if chunk:
        m["mask"] = {"size": chunk}
    ldim, lvdim, decay = right
    return {"type": "parallel", "mixer": {"left": m, "right": {"heads": len(decay), "dim": ldim, "vdim": lvdim, "decay": list(decay)}}, "mlp": mlp}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, shared=None):
    d = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def _model(vocab, width, layers, positions):
    d = {"architecture": "Putelix", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "layers": layers}
    if positions:
        d["max_positions"] = positions
    return d


CASES = {
    # (config, page size, rows of the distance tables). A: chunks longer and shorter than a page of 8, which part ways; a layer without
    # feed-forward; a shared expert of another width than the routed ones
    "A": (_model(83, 48, [_layer((6, 3, 16, 0.25, 8.0, 19, 15), (24, 16, (0.5, 0.9, 0.995)), _moe(6, 2, 40, 56)),
                          _layer((4, 2, 24, 0.2, 12.0, 40, 30), (16, 24, (0.97, 0.3)), _dense(72)),
                          _layer((3, 3, 16, 0.3, None, 5, 9), (8, 40, (0.8,)))], 320), 8, 12),
    # B: sizes that the tensor-core kernels take: heads of 64, 96 and 128, groups of 4, 1 and 2, memories of 64 to 128 entries
    "B": (_model(120, 64, [_layer((8, 2, 64, 0.125, 15.0, 48, 40), (64, 64, (0.6, 0.9, 0.99, 0.999)), _moe(8, 3, 48, 48)),
                           _layer((2, 2, 128, 0.1, 30.0, 130, 100), (128, 32, (0.95, 0.7)), _dense(96)),
                           _layer((4, 4, 96, 0.1, 10.0, 16, 14), (32, 96, (0.99,)), _moe(5, 2, 64)),
                           _layer((4, 1, 128, 0.12, 20.0, None, 64), (104, 8, (0.9, 0.999)))], 512), 16, 20),
    # C: sizes that take the kernels' slow paths (a width that is no multiple of 8, heads of 10 and 22, memories of 14 x 6 and 20 x 7), chunks
    # of a single position, one chosen expert, pages of 4
    "C": (_model(57, 44, [_layer((3, 1, 10, 0.35, 5.0, 1, 8), (14, 6, (0.9, 0.4)), _moe(4, 1, 20, 28)),
                          _layer((2, 2, 22, 0.25, 9.0, 33, 25), (20, 7, (0.99, 0.85, 0.2)), _dense(36))], 400), 4, 7),
    # D: one head, one expert layer whose tokens choose every expert, decays of 1 and 0, neither cap nor chunk in one layer, a chunk that
    # is a multiple of the page in the other; the checkpoint decides how many positions there are
    "D": (_model(64, 40, [_layer((1, 1, 32, 0.2, None, None, 70), (16, 16, (1.0, 0.0)), _moe(3, 3, 24, 24)),
                          _layer((4, 4, 16, 0.25, 6.0, 64, 50), (32, 32, (0.98,)), _moe(7, 5, 16))], None), 16, 16),
}

# float32: only the order of summation differs. bfloat16: activations are rounded to 8 bits between the kernels, and every sublayer's
# result is brought back to full size by its closing norm; a wrong key or a lost state moves the logits by 0.3 and more
LIMIT = {"float32": 3e-5, "bfloat16": 8e-2}
LENS = {"a": 150, "b": 67, "c": 41, "d": 9, "e": 118, "f": 2}


def make_folder(tmp: Path, name: str, store: str = "float32", std: float = 0.08, seed: int = 11, sharp: float = 1.0) -> Path:
    """A model folder for case ``name`` with random weights whose mechanisms all show: biases by distance and of the projections of
    size one half, position rows as large as the embedding, router logits far apart. ``sharp`` multiplies the query norms' weights, so
    that few keys matter and one that is lost, or seen when it should not be, moves the logits by far more than rounding does."""
    from llm_infrence_engine_b200.weights.random_init import random_tensors
    from llm_infrence_engine_b200.weights.safetensors_io import write_safetensors

    cfg, _, rel_rows = CASES[name]
    t = random_tensors(cfg, seed, std)
    g = torch.Generator().manual_seed(seed + 1)
    for key in t:
        if key == "pos" and not cfg.get("max_positions"):
            t[key] = torch.randn((333, cfg["width"]), generator=g) * 0.7
        elif key in ("embed", "pos"):
            t[key] = torch.randn(t[key].shape, generator=g) * 0.7
        elif key.endswith(".rel"):
            t[key] = torch.randn((rel_rows, t[key].shape[1]), generator=g) * 0.8
        elif key.endswith(".b"):
            t[key] = torch.randn(t[key].shape, generator=g) * 0.4
        elif key.endswith(".router"):
            t[key] = t[key] * 2.0
        elif key.endswith("left.q.norm"):
            t[key] = t[key] * 1.5 * sharp
        elif key.endswith("left.k.norm"):
            t[key] = t[key] * (1.0 + 0.5 * torch.randn(t[key].shape, generator=g))
    dtype = {"float32": torch.float32, "bfloat16": torch.bfloat16}[store]
    folder = Path(tmp) / f"putelix_{name}_{store}_{sharp}"
    folder.mkdir(parents=True, exist_ok=True)
    write_safetensors(folder / "model.safetensors", {k: v.to(dtype).contiguous() for k, v in t.items()})
    (folder / "config.json").write_text(json.dumps(cfg))
    return folder


def replayer(folder, name, dtype, max_tokens, kernels=None, device="cuda:0", **kw):
    from llm_infrence_engine_b200.engine import TraceReplayer

    return TraceReplayer(str(folder), dtype, max_tokens, device=device, kernels=kernels, block_size=CASES[name][1], **kw)


def plain_logits(cfg, tensors, tokens):
    return plain.forward(cfg, tensors, tokens, torch.float64)


class RouterTap:
    """Listens to the routers of a kernels object: what every call chose, in the order of the calls (a step calls once per layer with
    experts, with the step's rows)."""

    def __init__(self, kernels):
        self.K, self.calls = kernels, []
        inner = kernels.moe_router

        def listening(*args, **kw):
            out = inner(*args, **kw)
            self.calls.append(out[0].detach().cpu().long())
            return out

        kernels.moe_router = listening

    def close(self):
        del self.K.moe_router     # (the instance's attribute; the class's method is back)

    def choices(self, layers: int, rows_of: list, order: list) -> dict:
        """From the calls of a sequence of steps: per request, a list over the layers with experts of ``[T, top]``. ``rows_of[s]`` lists
        ``(request, rows)`` of step s in batch order."""
        out = {r: [[] for _ in range(layers)] for r in order}
        assert len(self.calls) == layers * len(rows_of), f"{len(self.calls)} router calls for {len(rows_of)} steps of {layers} layers"
        for s, step in enumerate(rows_of):
            for j in range(layers):
                ids, o = self.calls[s * layers + j], 0
                for rid, n in step:
                    out[rid][j].append(ids[o:o + n])
                    o += n
        return {r: [torch.cat(c) for c in per] for r, per in out.items()}


def moe_layers(cfg) -> int:
    return sum(1 for layer in cfg["layers"] if layer.get("mlp") and layer["mlp"]["kind"] == "moe")


def tapped_alone(rp, cfg, rid, tokens, cuts, step0=0):
    """``run_alone`` with the routers' choices: (logits [T, vocab], per layer with experts [T, top])."""
    tap = RouterTap(rp.runner.K)
    try:
        got = run_alone(rp, rid, tokens, cuts, step0)
    finally:
        tap.close()
    return got, tap.choices(moe_layers(cfg), [[(rid, hi - lo)] for lo, hi in cuts], [rid])[rid]


def judge(got, case, tokens, choices, dtype, what, own, limit=None):
    """The engine's logits against the oracle's. float32: against the oracle as it is. bfloat16: a router's choice between two nearly
    equal logits may fall the other way after rounding, which is no fault and changes the token's stream as a whole; so the oracle
    takes the experts that the engine took, and the engine's experts must be the router's own choice but where that hung on little
    (logits have a spread of about 3 here)."""
    folder, cfg, tensors = case[:3]
    limit = limit or LIMIT[dtype]
    want = own
    if dtype != "float32" and choices:
        regret = []
        want = plain.forward(cfg, tensors, tokens, torch.float64, forced=choices, regret_out=regret)[: got.shape[0]]
        worst = float(torch.stack(regret).max())
        assert worst <= 0.25, f"{what}: a router took an expert whose logit lies {worst:.3g} below its own choice"
    err = row_error(got, want)
    assert err <= limit, f"{what}: {err:.3g}"


def setup_case(tmp, name, dtype, lens=None, **kw):
    folder = make_folder(tmp, name, dtype, **kw)
    cfg, tensors = load_plain(folder)
    prompts = {k: prompt(cfg["vocab"], n, 3 + i) for i, (k, n) in enumerate((lens or LENS).items())}
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
            got, choices = tapped_alone(rp, cfg, f"{k}{n}", p, cuts, n)
            n += len(cuts)
            judge(got, case, p, choices, dtype, f"{name} {dtype} request {k} ({T} tokens) {what}", want[k])
            rp.cache.check_invariants()
    assert rp.cache.num_free_slots() == 4 and all(p.num_free == p.capacity for p in rp.cache.pools)


def check_mixed(case, name, dtype, kernels, device, seeds=(0, 1)):
    """Batches of unequal requests on a pool that holds only the live ones (pages and state slots are used again): every
    request as if it ran alone."""
    folder, cfg, tensors, prompts, want = case
    lens = {k: len(v) for k, v in prompts.items()}
    for seed in seeds:
        longest = sorted(lens.values(), reverse=True)
        rp = replayer(folder, name, dtype, sum(-(-n // 64) * 64 for n in longest[:4]), kernels, device)
        tap = RouterTap(rp.runner.K)
        got, rows_of = {k: [] for k in prompts}, []
        try:
            for n, step in enumerate(mixed_schedule(lens, seed)):
                entries = [{"id": rid, "tokens": prompts[rid][lo:hi], "want": list(range(hi - lo))} for rid, lo, hi in step]
                out = rp.step({"step": n, "entries": entries, "end": [rid for rid, lo, hi in step if hi == lens[rid]]})
                rp.cache.check_invariants()
                rows_of.append([(rid, hi - lo) for rid, lo, hi in step])
                o = 0
                for rid, lo, hi in step:
                    got[rid].append(out[o:o + hi - lo])
                    o += hi - lo
        finally:
            tap.close()
        choices = tap.choices(moe_layers(cfg), rows_of, list(prompts))
        for k in prompts:
            judge(torch.cat(got[k]), case, prompts[k], choices[k], dtype, f"{name} {dtype} mixed (seed {seed}) request {k}", want[k])
        assert rp.cache.num_free_slots() == 4 and all(p.num_free == p.capacity for p in rp.cache.pools)


def check_long_decoding(case, name, dtype, kernels, device, total=300):
    """A short prompt, then hundreds of tokens one by one: chunks begin and end on decoded tokens and give their pages back, and the
    memory of the first tokens fades or stays."""
    folder, cfg, tensors, prompts, want = case
    p = prompt(cfg["vocab"], total, 99)
    ref = plain_logits(cfg, tensors, p)
    rp = replayer(folder, name, dtype, 320, kernels, device)
    got, choices = tapped_alone(rp, cfg, "long", p, cuts_of(total, [3] + [1] * total))
    judge(got, case, p, choices, dtype, f"{name} {dtype} long decoding", ref)
    judge(got[:4], case, p, choices, dtype, f"{name} {dtype} first tokens", ref[:4])


def check_slot_reuse(case, name, dtype, kernels, device):
    """One request after another on the same slot, each beginning with a single token: the state of a request starts from zero and its
    positions from 0, whatever the slot's earlier owner left there."""
    folder, cfg, tensors, prompts, want = case
    rp = replayer(folder, name, dtype, 192, kernels, device)
    for n, (k, p) in enumerate(prompts.items()):
        p, ref = p[:12], want[k][:12]
        got, choices = tapped_alone(rp, cfg, f"s{n}", p, cuts_of(len(p), [1, 1, 2, 1, 3, 4]), 100 * n)
        judge(got, case, p, choices, dtype, f"{name} {dtype} request {k} on a used slot", ref)
