"""Putelix on the CPU: the plain implementation's mechanisms one by one, configuration, builder, weights, cache groups, and the
engine's host side (step building, pages, chunks, state slots, positions, scheduler) with the torch stand-in kernels, against the
plain implementation."""
import json
import math

import pytest
import torch

import plain_putelix as plain
from putelix_cases import CASES, check_long_decoding, check_mixed, check_slot_reuse, check_whole_and_cut, plain_logits, setup_case
from torch_kernels import TorchKernels

CPU_LENS = {"b": 67, "c": 41, "d": 9, "f": 2}


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("putelix")
    return {name: setup_case(tmp, name, "float32", CPU_LENS) for name in CASES}


# ------------------------------------------------------------------------------------------------ the plain implementation itself
def test_plain_norm_cap_and_activations_by_hand():
    x = torch.tensor([[3.0, -4.0]]).double()
    y = plain.rms_norm(x, torch.tensor([2.0, 0.5]).double(), 0.5)[0]
    f = 1 / math.sqrt(12.5 + 0.5)
    assert y.tolist() == pytest.approx([6 * f, -2 * f])
    assert plain.cap_tanh(x, 2.0)[0].tolist() == pytest.approx([2 * math.tanh(1.5), -2 * math.tanh(2.0)]) and plain.cap_tanh(x, None) is x
    W = {"p.up": torch.tensor([[1.0, 0.0], [0.0, 1.0]]).double(), "p.down": torch.tensor([[1.0, 1.0]]).double()}
    assert plain.dense_unit(W, "p", x).item() == pytest.approx(9.0)          # the negative entry is cut off


def test_plain_distance_rows_and_chunks_by_hand():
    # 8 rows: distances 0..3 have their own, then ln(n / 4) / ln(16) * 4 more, the last row from there on
    assert [plain.bucket(n, 8, 64.0) for n in (0, 1, 3, 4, 7, 8, 15, 16, 31, 32, 63, 64, 1000)] == [0, 1, 3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7]
    seen = plain.chunk_mask(7, 3)
    assert [row.nonzero()[:, 0].tolist() for row in seen] == [[0], [0, 1], [0, 1, 2], [3], [3, 4], [3, 4, 5], [6]]
    assert plain.chunk_mask(3, None).tolist() == torch.ones(3, 3).tril().bool().tolist()


def test_plain_attention_values_are_keys_before_the_norm():
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "scale": 0.5, "softcap": 1.0, "bias_max": 8, "mask": {"size": 4}}
    eye = torch.eye(2).double()
    W = {"p.q": eye, "p.k": 2 * eye, "p.q.b": torch.zeros(2), "p.k.b": torch.tensor([1.0, 0.0]), "p.q.norm": torch.tensor([1.0, 3.0]), "p.k.norm": torch.ones(2),
         "p.rel": torch.tensor([[0.25], [-1.0], [9.0], [9.0]]), "p.g": torch.tensor([[1.0, 0.0]]), "p.o": eye, "p.o.b": torch.tensor([0.0, 0.125])}
    W = {k: t.double() for k, t in W.items()}
    h = torch.tensor([[1.0, 0.0], [0.0, 2.0]]).double()
    out = plain.chunked_attention(m, W, "p", h, 0.0)
    k0, k1 = torch.tensor([3.0, 0.0]).double(), torch.tensor([1.0, 4.0]).double()      # 2 h + bias: the values, and the keys before their norm
    sig = 1 / (1 + math.exp(-1.0))
    assert out[0].tolist() == pytest.approx([3 * sig, 0.125])
    q1 = torch.tensor([0.0, 3 * math.sqrt(2.0)]).double()
    n0, n1 = k0 / math.sqrt(4.5), k1 / math.sqrt(8.5)
    s0, s1 = math.tanh(0.5 * float(q1 @ n0)) - 1.0, math.tanh(0.5 * float(q1 @ n1)) + 0.25
    a0 = math.exp(s0) / (math.exp(s0) + math.exp(s1))
    want = 0.5 * (a0 * k0 + (1 - a0) * k1)
    assert out[1].tolist() == pytest.approx([float(want[0]), float(want[1]) + 0.125])


def test_plain_linear_attention_by_hand():
    m = {"heads": 1, "dim": 1, "vdim": 2, "decay": [0.5]}
    W = {"p.q": torch.ones(1, 1), "p.k": torch.ones(1, 1), "p.v": torch.tensor([[1.0], [2.0]]), "p.g": torch.zeros(2, 1), "p.o": torch.eye(2), "p.norm": torch.tensor([1.0, 4.0])}
    W = {k: t.double() for k, t in W.items()}
    h = torch.tensor([[1.0], [2.0]]).double()
    out = plain.lightning_attention(m, W, "p", h, 1e-9)
    si = lambda z: z / (1 + math.exp(-z))
    S0 = [si(1) * si(1), si(1) * si(2)]
    S1 = [0.5 * S0[0] + si(2) * si(2), 0.5 * S0[1] + si(2) * si(4)]
    for row, S, q in ((out[0], S0, si(1)), (out[1], S1, si(2))):
        o = [q * s for s in S]
        f = 0.5 / math.sqrt((o[0] ** 2 + o[1] ** 2) / 2)
        assert row.tolist() == pytest.approx([o[0] * f, 4 * o[1] * f])


def test_plain_router_and_shared_gate_by_hand():
    ids, w = plain.route(torch.tensor([[1.0, 5.0, 3.0, -2.0]]).double(), 2)
    assert ids.tolist() == [[1, 2]] and w[0].tolist() == pytest.approx([1 / (1 + math.exp(-2.0)), 1 / (1 + math.exp(2.0))])
    one = torch.ones(1, 1).double()
    W = {"p.router": torch.zeros(2, 1).double(), "p.router.b": torch.tensor([0.0, 9.0]).double(), "p.shared.sg": one * math.log(3.0)}
    for e, f in (("e0", 5.0), ("e1", 1.0), ("shared", 2.0)):
        W.update({f"p.{e}.gate": one, f"p.{e}.up": one, f"p.{e}.down": f * one})
    got = plain.routed_experts({"router": {"experts": 2, "top": 1}, "shared": {"ff": 1}}, W, "p", one)
    s = 1 / (1 + math.exp(-1.0))
    assert got.item() == pytest.approx(s + 0.75 * 2 * s)         # the bias alone decides; sigmoid(ln 3) = 3/4


# ------------------------------------------------------------------------------------------------ configuration, builder, cache
def test_config_reads_every_key():
    from llm_infrence_engine_b200.config import ConfigError, PutelixConfig

    cfg = PutelixConfig.from_dict(CASES["A"][0])
    assert (cfg.vocab, cfg.width, cfg.eps, cfg.max_positions, len(cfg.layers)) == (83, 48, 1e-5, 320, 3)
    a, r, e = cfg.layers[0].mixer.left, cfg.layers[0].mixer.right, cfg.layers[0].mlp
    assert (a.heads, a.kv_heads, a.dim, a.scale, a.softcap, a.chunk, a.bias_max) == (6, 3, 16, 0.25, 8.0, 19, 15.0)
    assert (r.heads, r.dim, r.vdim, r.decay) == (3, 24, 16, (0.5, 0.9, 0.995)) and (e.experts, e.top, e.ff, e.shared_ff) == (6, 2, 40, 56)
    assert cfg.layers[1].mlp == 72 and cfg.layers[2].mlp is None and cfg.layers[2].mixer.left.softcap is None
    d = PutelixConfig.from_dict(CASES["D"][0])
    assert d.max_positions is None and d.layers[0].mixer.left.chunk is None and d.layers[1].mlp.shared_ff is None
    L = lambda d, i: d["layers"][i]["mixer"]
    for change in (lambda d: d["layers"][0].update(type="attention"), lambda d: L(d, 0)["left"].update(heads=4), lambda d: L(d, 0)["left"].update(vdim=8),
                   lambda d: L(d, 0)["left"].pop("bias_max"), lambda d: L(d, 0)["left"].update(softcap=0.0), lambda d: L(d, 0)["left"]["mask"].update(size=0),
                   lambda d: L(d, 0)["right"].update(decay=[0.5]), lambda d: L(d, 0)["right"].update(decay=[0.5, 0.5, 1.5]), lambda d: L(d, 0)["right"].update(dim=300),
                   lambda d: d["layers"][0]["mlp"].update(kind="other"), lambda d: d["layers"][0]["mlp"]["router"].update(top=7), lambda d: d.update(max_positions=0),
                   lambda d: d["norm"].update(eps=0.0), lambda d: d.update(layers=[])):
        bad = json.loads(json.dumps(CASES["A"][0]))
        change(bad)
        with pytest.raises(ConfigError):
            PutelixConfig.from_dict(bad)


def test_builder_names_the_checkpoint_tensors_and_the_cache():
    from llm_infrence_engine_b200.cache.spec import FixedStateSpec, PagedKVSpec
    from llm_infrence_engine_b200.engine.step import group_layout, has_fixed_state
    from llm_infrence_engine_b200.models import build_model_spec
    from llm_infrence_engine_b200.parts.base import ANY
    from llm_infrence_engine_b200.weights.loader import expected_tensors

    spec = build_model_spec(CASES["A"][0])
    want = {k: v[0] for k, v in expected_tensors(spec).items()}
    assert want["embed"] == (83, 48) and want["pos"] == (320, 48) and want["l0.mix.left.q.norm"] == (96,) and want["l0.mix.left.k.norm"] == (48,)
    assert want["l0.mix.left.rel"] == (ANY, 6) and want["l0.mix.left.o.b"] == (48,) and want["l0.mlp.shared.sg"] == (1, 48) and want["l0.mlp.router.b"] == (6,)
    assert want["l1.mlp.up"] == (72, 48) and want["l0.mix.right.norm"] == (48,) and want["l2.mix.right.v"] == (40, 48)
    assert {"l0.norm1", "l0.norm2", "l2.norm1", "final.norm", "l0.mlp.e5.down", "l0.mix.left.g", "l0.mix.right.g"} <= set(want)
    assert not any(n in want for n in ("head", "l0.mix.left.v", "l2.norm2", "l2.mlp.up", "l0.mlp.correction", "l0.mix.left.g.b"))
    specs = spec.cache_specs()
    assert specs[0] == (PagedKVSpec(3, 16, None, 0, 0, 19, token_scalar=True), FixedStateSpec((3, 16, 24)))
    assert specs[2] == (PagedKVSpec(3, 16, None, 0, 0, 5, token_scalar=True), FixedStateSpec((1, 40, 8)))
    groups, of_entry = group_layout(specs)
    assert len(groups) == 3 and of_entry == [(0, None), (1, None), (2, None)] and has_fixed_state(specs)
    assert {k: v[0] for k, v in expected_tensors(build_model_spec(CASES["D"][0])).items()}["pos"] == (ANY, 40)


def test_weights_load_and_biases_follow_their_rows(cases):
    from llm_infrence_engine_b200.models import build_model_spec
    from llm_infrence_engine_b200.weights import load_weights

    folder, cfg, t, _, _ = cases["C"]
    spec = build_model_spec(cfg)
    load_weights(spec, folder, torch.float32, "cpu")
    left, right = spec.layers[0].mixer.left, spec.layers[0].mixer.right
    assert left.w_qkv.shape == (48, 44) and left.b_qkv.shape == (48,)        # 30 + 10 + 3 rows of gates, padded to a multiple of 8
    assert torch.equal(left.b_qkv[:40], torch.cat([t["l0.mix.left.q.b"], t["l0.mix.left.k.b"]])) and float(left.b_qkv[40:].abs().max()) == 0.0
    assert torch.equal(left.w_qkv[40:43], t["l0.mix.left.g"])
    assert [left.rel_rows[n].item() for n in range(8)] == [plain.bucket(n, 7, 8) for n in range(8)]
    assert (right.q_col, right.k_col, right.v_col, right.g_col) == (0, 32, 64, 80) and torch.equal(right.w_in[64:76], t["l0.mix.right.v"])
    assert right.decay.tolist() == pytest.approx([0.9, 0.4])
    ff = spec.layers[0].ff
    assert torch.equal(ff.w_router, torch.cat([t["l0.mlp.router"], t["l0.mlp.shared.sg"]])) and torch.equal(ff.router_bias, t["l0.mlp.router.b"])
    d = build_model_spec(cases["D"][1])
    load_weights(d, cases["D"][0], torch.float32, "cpu")
    assert d.embedding.position_limit() == 333


def test_combinations_that_are_not_built_are_refused():
    from llm_infrence_engine_b200.parts import LinearRotary, MaskedAttention, PositionedEmbedding
    from llm_infrence_engine_b200.parts.mlp import RoutedExperts

    args = (16, 2, 1, 8, 8, 1.0, "p")
    for kw in (dict(values_are_keys=True), dict(qk_norm="rows", conv_taps=2), dict(qk_norm="rows", position=LinearRotary(8, 100.0)),
               dict(bias_far=9.0, scoring="sigmoid"), dict(bias_far=9.0, talking_heads=True)):
        with pytest.raises(ValueError):
            MaskedAttention(*args, **kw)
    with pytest.raises(ValueError):
        MaskedAttention(16, 2, 1, 8, 4, 1.0, "p", qk_norm="rows", values_are_keys=True)
    with pytest.raises(ValueError):
        RoutedExperts(16, 8, 4, 0, 2, "p", scoring="top_softmax")               # (a correction by default)
    with pytest.raises(ValueError):
        RoutedExperts(16, 8, 4, 0, 2, "p", correction=False, shared_gate="g")
    with pytest.raises(ValueError):
        PositionedEmbedding(8, 4, "e", "p", 16).add_into(None, None)


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


def test_what_a_fault_would_look_like(cases):
    """The oracle with one mechanism bent is far from itself: a chunk one longer, positions from 1, values taken after the norm's
    weight, a state that is lost after 20 tokens, and a gate or a bias left out all show far above the tests' limits."""
    folder, cfg, tensors, prompts, want = cases["A"]
    p = prompts["c"]

    def off(cfg2=None, **changed):
        return float((plain.forward(cfg2 or cfg, {**tensors, **changed}, p, torch.float64) - want["c"]).abs().max() / want["c"].std())

    longer = json.loads(json.dumps(cfg))
    longer["layers"][0]["mixer"]["left"]["mask"]["size"] += 1
    decays = json.loads(json.dumps(cfg))
    decays["layers"][0]["mixer"]["right"]["decay"][2] = 0.9
    assert off(longer) > 0.05 and off(decays) > 0.05
    assert off(pos=tensors["pos"].roll(-1, 0)) > 0.05
    for name in ("l0.mix.left.rel", "l0.mix.left.g", "l0.mix.left.k.b", "l0.mlp.router.b", "l0.mlp.shared.sg", "l1.mix.left.o.b"):
        assert off(**{name: torch.zeros_like(tensors[name])}) > 0.05, name
    assert off(**{"l0.mix.left.k.norm": torch.ones_like(tensors["l0.mix.left.k.norm"])}) > 0.05
    fresh = plain.forward(cfg, tensors, p[20:], torch.float64)
    assert float((fresh - want["c"][20:]).abs().max() / want["c"].std()) > 0.3


def test_a_request_longer_than_the_position_table_is_refused(cases):
    from llm_infrence_engine_b200.engine import Engine
    from putelix_cases import replayer

    folder, cfg, tensors, prompts, want = cases["A"]
    eng = Engine(folder, kernels=TorchKernels(), dtype="float32", device="cpu", max_len=4096, max_seqs=2, block_size=8, num_blocks=90)
    assert eng.config.max_len == 320 and eng.runner.max_len == 320
    with pytest.raises(ValueError):
        eng.generate([[1] * 310], max_new_tokens=20)
    rp = replayer(folder, "A", "float32", 640, TorchKernels(), "cpu")
    with pytest.raises(ValueError):
        rp.step({"step": 0, "entries": [{"id": "x", "tokens": [1] * 321, "want": [0]}], "end": []})


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
