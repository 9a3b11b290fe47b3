"""Sinorax on the CPU: the plain implementation's mechanisms one by one, configuration, builder, weights, cache groups, and the
engine's host side (step building, pages, windows, state slots, scheduler) with the torch stand-in kernels, against the plain
implementation."""
import json
import math

import pytest
import torch

import plain_sinorax as plain
from sinorax_cases import CASES, check_long_decoding, check_mixed, check_slot_reuse, check_whole_and_cut, plain_logits, setup_case
from torch_kernels import TorchKernels


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("sinorax")
    return {name: setup_case(tmp, name, "float32") for name in CASES}


# ------------------------------------------------------------------------------------------------ the plain implementation itself
def test_plain_dynamic_tanh_and_gelu_by_hand():
    W = {"n": torch.tensor([2.0, -1.0]).double(), "n.b": torch.tensor([0.5, 0.0]).double(), "n.alpha": torch.tensor(0.25).double()}
    y = plain.dynamic_tanh(torch.tensor([[4.0, -8.0]]).double(), W, "n")[0]
    assert y[0].item() == pytest.approx(2 * math.tanh(1.0) + 0.5) and y[1].item() == pytest.approx(math.tanh(2.0))
    z = torch.tensor([1.3]).double()
    assert plain.gelu_erf(z).item() == pytest.approx(1.3 * 0.5 * (1 + math.erf(1.3 / math.sqrt(2))))
    assert plain.cap_tanh(z, 2.0).item() == pytest.approx(2 * math.tanh(0.65)) and plain.cap_tanh(z, None) is z


def test_plain_bigram_rows():
    b = {"buckets": 10, "mul_prev": 3, "mul_cur": 7}
    assert plain.bigram_row(None, 4, b) == 10 and plain.bigram_row(5, 4, b) == (15 + 28) % 10
    cfg = {"embedding": {"bigram": b}}
    W = {"embed": torch.eye(6).double(), "bigram": torch.arange(11).double()[:, None].repeat(1, 6)}
    x = plain.embed(cfg, W, [2, 2, 5])
    assert [row[0].item() for row in x] == [10.0, (6 + 14) % 10, (6 + 35) % 10] and x[0, 2].item() == 11.0


def test_plain_values_turn_with_distance_only():
    """A key that owns the whole weight: the result is its value turned by (j - i), whatever i and j are by themselves."""
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 4, "scale": 1.0, "rot": {"dims": 2, "base": 100.0, "scaling": {"factor": 2.0}}}
    f = [1.0, 100.0 ** -0.5]
    v = torch.tensor([[1.0, 2.0, 3.0, 4.0]]).double()
    turned = plain.rotate_values(v.view(1, 1, 4).repeat(9, 1, 1), 100.0)
    back = plain.rotate_values(turned.roll(2, dims=0), 100.0, back=True)[8, 0]     # position 8 takes the value cached at position 6
    for k in (0, 1):
        a = -2 * f[k]
        u, w = v[0, k], v[0, k + 2]
        assert back[k].item() == pytest.approx((u * math.cos(a) - w * math.sin(a)).item())
        assert back[k + 2].item() == pytest.approx((w * math.cos(a) + u * math.sin(a)).item())
    q = plain.rotate_keys(torch.tensor([1.0, 0.0]).double().view(1, 1, 2).repeat(5, 1, 1), m["rot"])[4, 0]
    assert q[0].item() == pytest.approx(math.cos(2.0)) and q[1].item() == pytest.approx(math.sin(2.0))     # position 4, slowed down by 2


def test_plain_sigmoid_attention_by_hand():
    m = {"heads": 2, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 0.5, "mask": {"size": 2}}
    W = {"p.q": torch.tensor([[1.0], [2.0]]), "p.k": torch.ones(1, 1), "p.v": torch.ones(1, 1), "p.o": torch.eye(2), "p.r1": torch.tensor([0.0, 3.0]),
         "p.r2": torch.tensor([1.0, 0.5]), "p.pb": torch.tensor([0.0, -1.0])}
    W = {k: t.double() for k, t in W.items()}
    h = torch.tensor([[1.0], [2.0], [4.0]]).double()
    out = plain.sigmoid_attention(m, W, "p", h)

    def sig(z):
        return 1 / (1 + math.exp(-z))

    assert out[0].tolist() == pytest.approx([sig(0.5), sig(1.0 - 1.0)])
    # position 2 sees 1 and 2, not 0; head 1 loses 3 ln(1.5) at distance 1
    assert out[2].tolist() == pytest.approx([4 * sig(8.0) + 2 * sig(4.0), 4 * sig(16 - 1.0) + 2 * sig(8 - 3 * math.log(1.5) - 1.0)])


# ------------------------------------------------------------------------------------------------ configuration, builder, cache
def test_config_reads_every_key():
    from llm_infrence_engine_b200.config import ConfigError
    from llm_infrence_engine_b200.config.model_config import SinoraxConfig

    cfg = SinoraxConfig.from_dict(CASES["A"][0])
    assert (cfg.vocab, cfg.width, cfg.logit_scale, cfg.logit_softcap) == (83, 48, 0.7, 20.0)
    assert (cfg.bigram.buckets, cfg.bigram.mul_prev, cfg.bigram.mul_cur) == (61, 13, 5)
    s, t = cfg.layers[0], cfg.layers[1]
    assert (s.kind, s.mixer.heads, s.mixer.kv_heads, s.mixer.dim, s.mixer.vdim, s.mixer.scale, s.mixer.window, s.mixer.rot, s.ff) == ("attention_2", 6, 3, 16, 24, 0.25, 19, None, 56)
    assert (t.kind, t.mixer.vdim, t.mixer.window, t.mixer.rot.dims, t.mixer.rot.base, t.mixer.rot.factor) == ("attention", 16, None, 16, 900.0, 2.5)
    assert cfg.layers[2].ff is None and cfg.layers[3].mixer.rot.factor == 1.0
    c = SinoraxConfig.from_dict(CASES["C"][0])
    assert c.logit_scale == 1.0 and c.logit_softcap is None and SinoraxConfig.from_dict(CASES["D"][0]).bigram is None
    for change in (lambda d: d["layers"][0].update(type="attention_3"), lambda d: d["layers"][0]["mixer"].update(heads=4), lambda d: d["layers"][1]["mixer"].pop("rot"),
                   lambda d: d["layers"][1]["mixer"]["rot"].update(dims=26), lambda d: d["layers"][1]["mixer"]["rot"].update(dims=15),
                   lambda d: d["layers"][1]["mixer"].update(vdim=15), lambda d: d["layers"][0]["mixer"].update(rot={"dims": 2, "base": 10.0}),
                   lambda d: d["layers"][0].update(mlp={"kind": "moe", "ff": 8}), lambda d: d["embedding"]["bigram"].update(mul_cur=-1),
                   lambda d: d["layers"][1]["mixer"].update(mask={"size": 4}), lambda d: d.update(logit_softcap=-1.0)):
        bad = json.loads(json.dumps(CASES["A"][0]))
        change(bad)
        with pytest.raises(ConfigError):
            SinoraxConfig.from_dict(bad)


def test_builder_names_the_checkpoint_tensors_and_the_cache():
    from llm_infrence_engine_b200.cache.spec import FixedStateSpec, PagedKVSpec
    from llm_infrence_engine_b200.engine.step import group_layout, has_fixed_state
    from llm_infrence_engine_b200.models import build_model_spec
    from llm_infrence_engine_b200.weights.loader import expected_tensors

    spec = build_model_spec(CASES["A"][0])
    want = expected_tensors(spec)
    assert want["embed"][0] == (83, 48) and want["bigram"][0] == (62, 48) and want["head"][0] == (83, 48)
    assert want["l0.norm1.alpha"][0] == () and want["final.norm.b"][0] == (48,)
    assert {"l0.mix.r1", "l0.mix.r2", "l0.mix.pb", "l0.mix.q", "l0.mix.o", "l1.mix.q.b", "l1.mix.k.b", "l1.mix.v.b", "l1.mix.o.b", "l1.norm2b.alpha", "l0.mlp.up"} <= set(want)
    assert not any(n in want for n in ("l0.mix.q.b", "l0.mix.o.b", "l1.mix.r1", "l1.mix.pb", "l2.mlp.up", "l2.norm2", "l2.norm2b.b"))
    specs = spec.cache_specs()
    assert specs[:4] == [PagedKVSpec(3, 16, 19, 24), PagedKVSpec(2, 24, None, 16), PagedKVSpec(1, 32, 5, 32), PagedKVSpec(3, 16, None, 40)]
    assert specs[4] == FixedStateSpec((1,), zeroed=False) and len(specs) == 5      # a request's last token, behind the layers' entries
    groups, of_entry = group_layout(specs)
    assert len(groups) == 4 and of_entry == [0, 1, 2, 3, None] and has_fixed_state(specs)
    assert build_model_spec(CASES["D"][0]).cache_specs()[-1] == PagedKVSpec(1, 32, None, 32)


def test_weights_load_and_biases_follow_their_rows(tmp_path, cases):
    from llm_infrence_engine_b200.models import build_model_spec
    from llm_infrence_engine_b200.weights import load_weights

    folder, cfg, t, _, _ = cases["C"]
    spec = build_model_spec(cfg)
    load_weights(spec, folder, torch.float32, "cpu")
    m = spec.layers[0].mixer
    assert m.w_qkv.shape == (48, 44) and m.b_qkv.shape == (48,)        # 30 + 10 + 6 rows, padded to a multiple of 8
    assert torch.equal(m.b_qkv[:46], torch.cat([t["l0.mix.q.b"], t["l0.mix.k.b"], t["l0.mix.v.b"]])) and float(m.b_qkv[46:].abs().max()) == 0.0
    assert torch.equal(m.b_o, t["l0.mix.o.b"]) and spec.layers[0].norm1b.alpha.shape == ()
    assert torch.equal(spec.layers[1].mixer.pb, t["l1.mix.pb"]) and spec.layers[1].mixer.b_qkv is None
    assert torch.equal(spec.embedding.bigram, t["bigram"]) and torch.equal(spec.head.matrix(), t["head"])


def test_a_looped_model_refuses_a_bigram_embedding():
    from llm_infrence_engine_b200.parts import BigramEmbedding

    with pytest.raises(ValueError):
        BigramEmbedding(8, 4, "e", "b", 3, 1, 1).add_into(None, None)
    with pytest.raises(ValueError):
        BigramEmbedding(8, 4, "e", "b", 0, 1, 1)


# ------------------------------------------------------------------------------------------------ the engine's host side
@pytest.mark.parametrize("name", sorted(CASES))
def test_engine_whole_and_cut_on_cpu(cases, name):
    check_whole_and_cut(cases[name], name, "float32", TorchKernels(), "cpu", only=("b", "d", "f"))


def test_engine_mixed_batches_on_cpu(cases):
    check_mixed(cases["C"], "C", "float32", TorchKernels(), "cpu", seeds=(0,))


def test_engine_long_decoding_on_cpu(cases):
    check_long_decoding(cases["A"], "A", "float32", TorchKernels(), "cpu", total=60)


def test_first_tokens_on_used_slots_on_cpu(cases):
    check_slot_reuse(cases["A"], "A", "float32", TorchKernels(), "cpu")


def test_a_lost_previous_token_shows(cases):
    """The oracle without its bigram rows, or with the previous token forgotten at a cut, is far from the engine's logits."""
    folder, cfg, tensors, prompts, want = cases["A"]
    p = prompts["c"]
    W = dict(tensors)
    W["bigram"] = torch.zeros_like(W["bigram"])
    without = plain.forward(cfg, W, p, torch.float64)
    assert float((without - want["c"]).abs().max()) > 0.3 * float(want["c"].std())


def test_greedy_generation_through_the_entry_point_on_cpu(cases):
    from llm_infrence_engine_b200.engine import Engine

    folder, cfg, tensors, prompts, want = cases["C"]
    eng = Engine(folder, kernels=TorchKernels(), dtype="float32", device="cpu", max_len=128, max_seqs=3, block_size=16, num_blocks=20,
                 max_num_batched_tokens=24)
    ps = [prompts["c"], prompts["d"], prompts["f"], prompts["b"][:30]]
    results = eng.generate(ps, max_new_tokens=8)
    for p, r in zip(ps, results):
        seq = list(p) + r.token_ids
        ref = plain_logits(cfg, tensors, seq)[len(p) - 1:-1]
        assert r.token_ids == ref.argmax(-1).tolist()
    eng.cache.check_invariants()
    assert all(pool.num_free == pool.capacity for pool in eng.cache.pools)
