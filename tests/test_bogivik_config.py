"""Bogivik on the host: config.json to the model's description, tensor names, cache and state needs, errors; pages of a cache
that keeps chunks; the plain implementation's own mechanisms against each other."""
import copy
import json
import math
import os

import pytest
import torch

import bogivik_tiny as BT
from plain import bogivik_plain as BP
from zedinfer_b200.cache import CacheManager, StateNeed
from zedinfer_b200.cache.manager import PagedKVNeed
from zedinfer_b200.config.registry import ConfigError, load_model_config, resolve_architecture
from zedinfer_b200.engine.model import Model

F64 = torch.float64


def spec_of(raw):
    arch = resolve_architecture(raw)
    spec = arch.build_spec(arch.parse(raw))
    spec.validate()
    return spec


def test_the_architecture_is_found_by_its_name():
    assert resolve_architecture({"architecture": "Bogivik"}).name == "Bogivik"
    assert resolve_architecture({"model_type": "bogivik"}).name == "Bogivik"
    libs = resolve_architecture({"architecture": "Bogivik"}).kernel_libraries
    assert "linrec" in libs and "rowwise" in libs


def test_layers_and_their_parts():
    spec = spec_of(BT.BG_A)
    assert [l.block for l in spec.layers] == ["shared_norm"] * 5
    assert [(l.mixer.kind, l.extra["mixer2"][1].kind if "mixer2" in l.extra else None, l.ffn.kind if l.ffn else None) for l in spec.layers] == [
        ("normed_attention", "exp_gate", "gated_mlp"), ("normed_attention", None, "gated_mlp"), ("normed_attention", "exp_gate", None),
        ("normed_attention", None, "gated_mlp"), ("normed_attention", None, None)]
    left, att = spec.layers[0].mixer.params, spec.layers[1].mixer.params
    assert (left["num_heads"], left["num_kv_heads"], left["head_dim"], left["v_head_dim"], left["chunk"], left["scale"]) == (4, 2, 32, 16, 13, 0.2)
    assert left["qk_norm"] == "head" and left["qkv_bias"] and left["out_bias"] and left["gate"]
    pos = left["position"].params
    assert pos["interleaved"] and pos["dims"] == 16 and pos["theta"] == 5000.0 and pos["scaling"]["original"] == 64.0
    assert att["qk_norm"] == "row" and att["heat"] == (0.4, 16.0) and att["bias_rows"] == 16 and att["bias_max"] == 40.0
    # the first v_mix layer is the first in the run order that says so, whatever stands before it
    assert [l.mixer.params.get("value_mix") for l in spec.layers] == [None, "first", None, "mix", None]
    assert spec.layers[1].ffn.params["activation"] == "gelu_tanh"
    right = spec.layers[2].extra["mixer2"][1].params
    assert (right["heads"], right["dim"], right["vdim"], right["gate_cap"]) == (2, 24, 8, 12.0)
    assert sorted(spec.layers[0].norms) == ["mix2_out", "mix_out", "norm1"] and sorted(spec.layers[1].norms) == ["norm1"]
    assert not spec.tie_word_embeddings


def test_tensor_names_and_a_size_that_only_a_shape_gives(tmp_path):
    names = Model(spec_of(BT.BG_A)).tensor_specs()
    assert names["l1.mix.rel"].shape == (16, 4) and names["l1.mix.vmix"].shape == () and names["l3.mix.vmix"].shape == ()
    assert names["l1.mix.q.norm"].shape == (64,) and names["l1.mix.k.norm"].shape == (32,) and names["l0.mix.left.q.norm"].shape == (32,)
    assert names["l0.mix.left.o.b"].shape == (96,) and names["l0.mix.left.g"].shape == (64, 96) and names["l0.mix.right.i.b"].shape == (3,)
    assert names["l0.mix.right.norm"].shape == (72,) and names["l0.mix.left.out"].shape == (96,) and names["head"].shape == (211, 96)
    for absent in ("l1.mix.q.b", "l4.mix.vmix", "l2.mlp.up", "l0.norm2", "l0.mix.left.rel", "l1.mix.o.b"):
        assert absent not in names
    # the folder's config.json need not name the number of buckets: the table's shape gives it
    out = BT.make_model_dir(tmp_path, "A")
    path = os.path.join(out, "config.json")
    raw = json.load(open(path))
    for layer in raw["layers"]:
        layer["mixer"].pop("bias_rows", None)
    json.dump(raw, open(path, "w"))
    _, _, spec = load_model_config(out)
    assert [l.mixer.params.get("bias_rows") for l in spec.layers] == [None, 16, None, 8, 6]


def test_caches_and_states():
    model = Model(spec_of(BT.BG_A))
    needs = dict(model.cache_needs())
    assert needs[0] == PagedKVNeed(2, 32, None, chunk=13) and needs[1] == PagedKVNeed(2, 24, None)
    assert needs[2] == PagedKVNeed(2, 40, None, chunk=29)
    # per head: vdim columns and the key sum, of dim entries and a running maximum each
    assert needs[(0, "mixer2")] == StateNeed((3 * 25 * 17,), torch.float32)
    assert model.capture_safe()
    assert len(CacheManager(list(needs.items()), 4, max_requests=3).groups) == 5
    assert dict(Model(spec_of(BT.BG_E)).cache_needs())[1] == PagedKVNeed(1, 8, None)            # no mask: every key
    assert CacheManager(list(Model(spec_of(BT.BG_D)).cache_needs()), 16, max_requests=2).slots.num_slots == 0


@pytest.mark.parametrize("chunk,page", [(10, 4), (8, 4), (3, 8), (1, 4), (64, 16)])
def test_pages_of_chunks_are_given_back_when_a_new_chunk_opens(chunk, page):
    """Whatever the portions: the pages that are kept hold every key of the next query's chunk, and none lies wholly before
    it; under a bound on a step's tokens the pool is as small as that allows and never runs out."""
    bound = 7
    cache = CacheManager([(0, PagedKVNeed(1, 8, None, chunk=chunk))], page, max_requests=2, max_step_tokens=bound)
    cache.set_num_pages(1000)
    assert cache.groups[0].num_pages == min(1000, 2 * ((chunk + bound + page - 2) // page + 1)) and cache.step_bound == bound
    rcs = [cache.open("a"), cache.open("b")]
    g = torch.Generator().manual_seed(chunk)
    for _ in range(120):
        rc = rcs[int(torch.randint(2, (1,), generator=g))]
        n = int(torch.randint(1, bound + 1, (1,), generator=g))
        cache.ensure(rc, rc.length + n)
        start = rc.length // chunk * chunk                                   # what the step's first query reads from
        table = rc.tables[0]
        assert all(table[b] >= 0 for b in range(start // page, (rc.length + n - 1) // page + 1))
        cache.commit(rc, rc.length + n)
        first = rc.length // chunk * chunk
        assert all((p >= 0) == (b >= first // page) for b, p in enumerate(rc.tables[0]))
        cache.check()
    for rc in rcs:
        cache.close(rc)
    assert cache.groups[0].pool.num_used == 0
    with pytest.raises(ValueError):
        CacheManager([(0, PagedKVNeed(1, 8, 5, chunk=5))], 4)
    # layers with other chunks, or with a window of that size, have pools of their own
    three = CacheManager([(0, PagedKVNeed(1, 8, None, chunk=8)), (1, PagedKVNeed(1, 8, 8)), (2, PagedKVNeed(1, 8, None, chunk=9)),
                          (3, PagedKVNeed(1, 8, None, chunk=8))], 4)
    assert [g.calls for g in three.groups] == [[0, 3], [1], [2]]


@pytest.mark.parametrize("edit,word", [
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c["layers"][0].update(type="delta"), "type"),
    (lambda c: c["layers"][1]["mixer"].update(heads=3), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"].update(bias_max=8), "bias_max"),
    (lambda c: c["layers"][1]["mixer"].pop("bias_max"), "bias_max"),
    (lambda c: c["layers"][1]["mixer"].update(scale=0), "scale"),
    (lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=0), "every"),
    (lambda c: c["layers"][1]["mixer"].update(v_mix=1), "v_mix"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=20), "v_mix"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("high"), "high"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(mask={"size": 0}), "mask"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("gate_cap"), "gate_cap"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][1]["mlp"].update(kind="moe"), "mlp"),
    (lambda c: c["layers"][1]["mlp"].update(ff=0), "ff"),
])
def test_errors_name_the_key(edit, word):
    cfg = copy.deepcopy(BT.BG_A)
    edit(cfg)
    with pytest.raises(ConfigError) as e:
        spec_of(cfg)
    assert word in str(e.value)


@pytest.mark.parametrize("rows,farthest", [(16, 40), (2, 5), (32, 1000), (12, 30), (8, 100.5), (8, 4096), (6, 9), (2, 1.5)])
def test_distances_and_their_buckets(rows, farthest):
    from zedinfer_b200.parts.normed_attention import distance_buckets
    got = distance_buckets(rows, farthest)
    assert got == [BP.distance_bucket(n, rows, farthest) for n in range(len(got))] and got == sorted(got)
    assert got[-1] == rows - 1 and got[:rows // 2] == list(range(rows // 2))
    assert all(BP.distance_bucket(n, rows, farthest) == rows - 1 for n in (len(got), len(got) + 1, 10 ** 6))


def test_a_distance_on_a_buckets_edge_opens_it():
    """4 * 2^(k / 2): with 8 rows and the farthest distance 16, distances 8 and 16 are edges; with 20 rows and 320 the distances
    20, 40 and 160 are, where the quotient of two rounded logarithms may fall short of the whole number."""
    from zedinfer_b200.parts.normed_attention import distance_bucket
    assert [distance_bucket(n, 8, 16) for n in (4, 7, 8, 15, 16)] == [4, 5, 6, 7, 7]
    assert [distance_bucket(n, 20, 320) for n in (19, 20, 39, 40, 159, 160)] == [11, 12, 13, 14, 17, 18]


@pytest.mark.parametrize("dims,base,scaling", [(32, 10000.0, (8.0, 1.0, 4.0, 512)), (8, 100.0, (4.0, 1.0, 2.0, 30)), (64, 5e5, (2.0, 2.0, 8.0, 100))])
def test_frequencies_stretched_by_wavelength(dims, base, scaling):
    from zedinfer_b200.parts import SpanRotaryPosition
    sc = dict(zip(("factor", "low", "high", "original"), scaling))
    rule = SpanRotaryPosition(dims, dims, base, interleaved=True, scaling=sc)
    ref = torch.tensor(BP.turn_frequencies(dims, base, sc), dtype=F64)
    plain = torch.tensor(BP.turn_frequencies(dims, base, None), dtype=F64)
    assert torch.allclose(rule.inverse_frequencies().double(), ref, rtol=1e-6) and rule.magnitude == 1.0
    ratio = ref / plain
    kept, slowed = ratio == 1.0, torch.isclose(ratio, torch.tensor(1.0 / scaling[0], dtype=F64))
    assert bool(kept.any()) and bool(slowed.any()) and bool((~kept & ~slowed).any())         # the premise: all three cases occur


def test_the_plain_mechanisms_agree_with_one_another():
    """The memory walked in two pieces from the state between them; its gates at their extremes; values mixed by 0 and 1; a
    prefix's logits do not depend on what follows; a chunk's first token sees itself alone."""
    g = torch.Generator().manual_seed(0)
    n, H, d, dv = 9, 2, 6, 5
    q, k, v = (torch.randn(n, H, w, generator=g, dtype=F64) for w in (d, d, dv))
    i, f = torch.randn(n, H, generator=g, dtype=F64) * 4, -torch.rand(n, H, generator=g, dtype=F64) * 3
    whole, end = BP.exponential_gate_walk(q, k, v, i, f)
    a, mid = BP.exponential_gate_walk(q[:4], k[:4], v[:4], i[:4], f[:4])
    b, end2 = BP.exponential_gate_walk(q[4:], k[4:], v[4:], i[4:], f[4:], mid)
    assert torch.allclose(torch.cat([a, b]), whole) and all(torch.allclose(x, y) for x, y in zip(end, end2))
    # in another arrangement of the same sums, without a running maximum: weights e^(i_s + sum of f behind s)
    cum = torch.cumsum(f, 0)
    for t in range(n):
        wts = torch.exp(i[:t + 1] + cum[t] - cum[:t + 1])                                       # [t + 1, H]
        dots = (k[:t + 1] * q[t]).sum(-1) * wts
        num, den = torch.einsum("sh,shv->hv", dots, v[:t + 1]), dots.sum(0).abs()
        m = torch.zeros(H, dtype=F64)
        for s in range(t + 1):
            m = torch.maximum(f[s] + m, i[s])
        ref = num * torch.exp(-m)[:, None] / (torch.maximum(den * torch.exp(-m), torch.exp(-m)) + BP.READ_OUT_EPS)[:, None]
        assert torch.allclose(whole[t], ref, atol=1e-10)
    first = torch.randn(3, 4, dtype=F64)
    assert torch.equal(BP.mixed_values(torch.zeros(3, 4, dtype=F64), first, 1.0), first) and BP.mixed_values(first, None, 1.0) is first
    assert BP.query_temperature(14, 0.5, 16) == 1.0 and math.isclose(BP.query_temperature(15, 0.5, 16), 1.0 + 0.5 * math.log(2.0))
    assert BP.query_temperature(0, 0.5, 1) == 1.0 + 0.5 * math.log(2.0)
    cfg = BT.BG_C
    from zedinfer_b200.weights.random_init import random_tensors
    names = Model(spec_of(cfg)).tensor_specs()
    wts = {k: v.double() for k, v in random_tensors(names, 3, torch.float32, init_scale=5.0).items()}
    toks = [5, 17, 3, 99, 140, 2, 2, 60]
    whole = BP.forward(cfg, wts, toks)
    assert torch.allclose(BP.forward(cfg, wts, toks[:5]), whole[:5], atol=1e-9)
