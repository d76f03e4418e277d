"""Bogivik in the engine against the plain implementation (tests/plain/bogivik_plain.py): every mechanism alone, then whole
models under every way of cutting the work, long decoding, generation through the Python entry point, the trace program and
the command-line programs."""
import json
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

import bogivik_tiny as BT
import traces
from part_util import DEV, bind_random, feed, rel_err
from plain import bogivik_plain as BP
from replay_util import run_trace

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F64 = torch.float64
BOTH = [torch.float32, torch.bfloat16]


def tol_for(dtype):
    return 2e-4 if dtype in ("float32", torch.float32) else 6e-2


def tol_part(dtype, f32=3e-5, bf16=5e-2):
    return f32 if dtype == torch.float32 else bf16


# ---------------------------------------------------------------------------------------------
# kernels alone
# ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("rows,hidden", [(1, 40), (7, 96), (33, 1536), (5, 73), (3, 52), (4, 2560), (2, 5120)])
def test_branches_that_join_the_stream_together(dtype, rows, hidden):
    """h += y + f, out = U(h) w: both branches, either alone, none; two outputs joined on the way (one so small that the epsilon
    shows); partial sums; chosen rows, which leave the stream as it is."""
    from zedinfer_b200 import ops
    g = torch.Generator().manual_seed(rows * 1000 + hidden)
    h0 = torch.randn(rows, hidden, generator=g) * 2
    y, f = (torch.randn(rows, hidden, generator=g).to(dtype) for _ in range(2))
    y2 = (torch.randn(rows, hidden, generator=g) * 2e-3).to(dtype)
    w, w1, w2 = (1 + 0.3 * torch.randn(hidden, generator=g) for _ in range(3))
    eps, jeps = 1e-5, 1e-6
    idx = torch.tensor([rows - 1, 0, rows // 2], dtype=torch.int32)
    joined = 0.5 * (BP.rms_unit(y.double(), jeps) * w1.double() + BP.rms_unit(y2.double(), jeps) * w2.double())
    assert float((BP.rms_unit(y2.double(), 0.0) - BP.rms_unit(y2.double(), jeps)).abs().max()) > 0.05      # premise: epsilon shows
    parts = torch.randn(3, rows, hidden, generator=g)
    cases = [(y, f, None, y.double() + f.double()), (y, None, None, y.double()), (None, f, None, f.double()), (None, None, None, 0.0),
             (y, f, (y2, w1, w2, jeps), joined + f.double()), (y, None, (y2, w1, w2, jeps), joined),
             (y, parts, None, y.double() + parts.sum(0).to(dtype).double()), (parts, f, None, parts.sum(0).to(dtype).double() + f.double())]
    dev = lambda t: None if t is None else t.to(DEV)
    for y_in, f_in, join, add in cases:
        want = h0.double() + add
        normed = BP.rms_unit(want, eps) * w.double()
        jd = tuple(dev(t) if torch.is_tensor(t) else t for t in join) if join else None
        loose = 1e-2 if (dtype == torch.bfloat16 and any(t is parts for t in (y_in, f_in))) else 3e-6     # the sums' own rounding
        h, out = h0.clone().to(DEV), torch.empty(rows, hidden, dtype=dtype, device=DEV)
        ops.branches_rmsnorm(h, dev(y_in), dev(f_in), w.to(DEV), eps, out, join=jd)
        assert rel_err(h, want) < loose and rel_err(out, normed) < tol_part(dtype, 3e-6, 2e-2)
        h, out = h0.clone().to(DEV), torch.empty(3, hidden, dtype=dtype, device=DEV)
        ops.branches_rmsnorm(h, dev(y_in), dev(f_in), w.to(DEV), eps, out, row_idx=idx.to(DEV), join=jd)
        assert torch.equal(h.cpu(), h0) and rel_err(out, normed[idx.long()]) < tol_part(dtype, 3e-6, 2e-2)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("rows", [1, 5, 12, 40, 150, 300])
@pytest.mark.parametrize("hidden,ff", [(64, 80), (160, 224), (52, 36), (96, 40)])
def test_gated_gelu_feed_forward(dtype, rows, hidden, ff):
    """On the weight-streaming kernel, the library product and the tensor-core kernel with the activation in its epilogue; inputs
    so large that the tanh form and the exact one, and both ends of the function, are told apart."""
    from zedinfer_b200.parts import GatedMLP
    part = GatedMLP(hidden, ff, activation="gelu_tanh", names={"gate": "gate", "up": "up", "down": "down"})
    t = bind_random(part, dtype, seed=ff, scale=0.3)
    x = torch.randn(rows, hidden, generator=torch.Generator().manual_seed(rows)).to(dtype)
    got = part.forward(x.to(DEV), _bare_context(rows, dtype))
    assert rel_err(got, BP.gelu_ff(x.double(), t, "")) < tol_part(dtype, 3e-5, 3e-2)
    with pytest.raises(ValueError):
        GatedMLP(8, 8, activation="gelu")


def _bare_context(n, dtype):
    from zedinfer_b200.parts import StepContext
    dev = torch.device(DEV)
    z = torch.zeros(n, dtype=torch.int32, device=dev)
    return StepContext(n_tokens=n, n_segments=1, dtype=dtype, device=dev, token_ids=z, positions=z, tok_seg=z, tables=[], slots=None,
                       seg_start_host=[0], seg_len_host=[n], seg_pos0_host=[0], slots_host=[-1])


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("heads,dim,vdim,cap", [(4, 16, 24, 6.0), (3, 136, 12, 15.0), (2, 72, 8, 1.0), (1, 8, 136, 12.0), (6, 40, 20, 30.0), (2, 200, 17, 5.0),
                                                (5, 4, 1, 4.0), (3, 64, 64, 10.0), (2, 128, 128, 8.0)])
def test_the_matrix_memory_walked_in_two_forms(dtype, heads, dim, vdim, cap):
    """Three segments of unequal length (one of a single token, one that starts from a state the slot already holds, one without a
    slot) through the walk that makes its own inputs ready and through the one that finds them made ready: both equal the plain
    walk and leave the same state (matrix, key sum, running maximum) behind, and they equal each other bit by bit."""
    from zedinfer_b200 import ops
    g0 = torch.Generator().manual_seed(dim * 7 + vdim)
    lens = [37, 1, 70]
    n = sum(lens)
    q, k = (torch.randn(n, heads * dim, generator=g0).to(dtype) for _ in range(2))
    v = torch.randn(n, heads * vdim, generator=g0).to(dtype)
    a, b = ((torch.randn(n, heads, generator=g0) * 4).to(dtype) for _ in range(2))
    bi, bf = torch.randn(heads, generator=g0) * 2, torch.randn(heads, generator=g0) + 2
    rows, width = vdim + 1, heads * (vdim + 1) * (dim + 1)
    assert ops.linear_state_floats("expgate", heads, dim, vdim) == width
    bounds = torch.tensor([[0, 37], [37, 38], [38, n]], dtype=torch.int32, device=DEV)
    slots = torch.tensor([2, -1, 0], dtype=torch.int32, device=DEV)
    qd, kd, vd = q.double().view(n, heads, dim) * dim ** -0.5, k.double().view(n, heads, dim), v.double().view(n, heads, vdim)
    li = cap * torch.tanh((a.double() + bi.double()) / cap)
    lf = torch.nn.functional.logsigmoid(cap * torch.tanh((b.double() + bf.double()) / cap))
    S0, n0, m0 = torch.randn(heads, dim, vdim, generator=g0) * 0.2, torch.randn(heads, dim, generator=g0) * 0.2, torch.randn(heads, generator=g0)
    refs, ends, at = [], [], 0
    for i, ln in enumerate(lens):
        sl = slice(at, at + ln)
        o, e = BP.exponential_gate_walk(qd[sl], kd[sl], vd[sl], li[sl], lf[sl], (S0.double(), n0.double(), m0.double()) if i == 2 else None)
        refs.append(o), ends.append(e)
        at += ln
    ref = torch.cat(refs)
    results = []
    for with_work in (False, True):
        state = torch.full((3, width + 11), 7.0, device=DEV)
        state[2, :width] = 0.0
        state[0, :heads * rows * dim] = torch.cat([S0.transpose(1, 2), n0[:, None]], dim=1).reshape(-1).to(DEV)
        state[0, heads * rows * dim:width] = m0[:, None].expand(heads, rows).reshape(-1).to(DEV)
        y, den = torch.empty(n, heads * vdim, dtype=torch.float32, device=DEV), torch.empty(n, heads, dtype=torch.float32, device=DEV)
        work = torch.empty(ops.linear_state_work_floats("expgate", n, heads, dim, vdim), dtype=torch.float32, device=DEV) if with_work else None
        ops.linear_state("expgate", q.to(DEV), k.to(DEV), v.to(DEV), state, slots, bounds, y, 3, heads, heads, dim, vdim, a=a.to(DEV), b=b.to(DEV),
                         dt_bias=bi.to(DEV), a_log=bf.to(DEV), q_scale=dim ** -0.5, den=den, gate_cap=cap, work=work)
        got = y.view(n, heads, vdim).double().cpu() / den.double().cpu()[..., None]
        # the inputs are what they are in either type; where n . q nearly cancels, its float32 sum is divided by
        assert rel_err(got, ref) < 3e-4 and float((got - ref).abs().median()) < 1e-6, with_work
        for slot, end in ((2, ends[0]), (0, ends[2])):
            cols = state[slot, :heads * rows * dim].view(heads, rows, dim).cpu()
            maxima = state[slot, heads * rows * dim:width].view(heads, rows).cpu()
            assert rel_err(cols[:, :vdim].transpose(1, 2), end[0]) < 2e-5 and rel_err(cols[:, vdim], end[1]) < 2e-5
            assert rel_err(maxima, end[2][:, None].expand(heads, rows)) < 1e-5
        assert bool((state[:, width:] == 7.0).all()) and bool((state[1] == 7.0).all())        # nothing else is touched
        results.append((y.clone(), den.clone(), state.clone()))
    assert all(torch.equal(x, z) for x, z in zip(*results))


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("inner,groups,wlen", [(48, 4, 48), (96, 1, 96), (1200, 3, 1200), (20, 20, 1), (1536, 12, 1536), (2048, 4, 512), (520, 2, 520), (4096, 4, 4096)])
def test_unit_groups_of_a_quotient(dtype, inner, groups, wlen):
    """Every group divided by its own number first: it shows through the epsilon alone, so some numbers are large."""
    from zedinfer_b200 import ops
    g = torch.Generator().manual_seed(inner)
    n, eps = 5, 1e-5
    y, z = torch.randn(n, inner, generator=g) * 3, torch.randn(n, inner, generator=g).to(dtype)
    den = torch.exp(torch.randn(n, groups, generator=g) * 3 + 4)
    w = (1 + 0.2 * torch.randn(wlen, generator=g)).to(dtype)
    for gate in ("sigmoid", "silu", None):
        for d in (den, None):
            out = torch.empty(n, inner, dtype=dtype, device=DEV)
            ops.group_rmsnorm_gate(y.to(DEV), z.to(DEV) if gate else None, w.to(DEV), groups, eps, out, gate=gate, den=None if d is None else d.to(DEV))
            o = y.double().view(n, groups, -1) / (1.0 if d is None else d.double()[..., None])
            ref = BP.rms_unit(o, eps).view(n, inner) * w.double().repeat(inner // wlen)
            if gate:
                ref = ref * BP.logistic(z.double()) * (z.double() if gate == "silu" else 1.0)
            assert rel_err(out, ref) < tol_part(dtype, 3e-6, 1e-2)


# ---------------------------------------------------------------------------------------------
# mixers alone
# ---------------------------------------------------------------------------------------------
SCHEDULE_ABC = [[("a", 6), ("b", 2)], [("b", 1), ("a", 1)], [("a", 1)], [("a", 2), ("b", 7), "end:b"], [("c", 3), ("a", 20)],
                [("c", 1), ("a", 1)], [("c", 8), ("a", 14)]]
SCHEDULE_AB = [[("a", 9), ("b", 2)], [("b", 1), ("a", 1)], [("a", 1)], [("a", 33), ("b", 15)], [("b", 1)], [("a", 2)], [("a", 15)]]


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("heads,dim,vdim,cap", [(3, 16, 24, 6.0), (1, 40, 20, 2.0), (4, 8, 136, 12.0), (2, 136, 16, 15.0), (9, 40, 64, 9.0), (1, 256, 4, 5.0), (2, 12, 1, 7.0)])
def test_exponential_gate_mixer_over_portions_and_slots_used_again(dtype, heads, dim, vdim, cap):
    """Two requests in shared steps, cut down to single tokens, then a third in the slot the second gave back: it starts from zeros,
    the running maximum included."""
    from zedinfer_b200.cache import CacheManager
    from zedinfer_b200.parts import ExpGateMixer
    hidden, eps = 64, 1e-5
    mixer = ExpGateMixer(hidden, heads, dim, vdim, cap, eps)
    over = {"norm": 1 + 0.1 * torch.randn(heads * vdim), "i.b": torch.linspace(-2.0, 3.0, heads), "f.b": torch.linspace(4.0, -1.0, heads)}
    t = bind_random(mixer, dtype, seed=dim, scale=0.3, overrides=over)
    cache = CacheManager([(0, mixer.cache_need())], 16, max_requests=2)
    cache.allocate_device(1, dtype, DEV)
    g = torch.Generator().manual_seed(6)
    xs = {r: torch.randn(n, hidden, generator=g).to(dtype) for r, n in (("a", 45), ("b", 10), ("c", 12))}
    got, = feed([mixer], [cache.view_for_call(0)], cache, dtype, xs, SCHEDULE_ABC)
    m = {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}
    for rid, x in xs.items():
        if dtype == torch.float32:
            assert rel_err(got[rid], BP.matrix_memory(x.double(), t, "", m, eps)) < 1e-4, rid
        else:
            # a head whose read-out happens to be small magnifies the projections' rounding (its root mean square divides it):
            # the typical entry is held tightly, the worst loosely
            d = (got[rid].double() - BP.matrix_memory(x.double(), t, "", m, eps)).abs()
            size = max(1.0, float(got[rid].abs().max()))
            assert float(d.median()) < 2e-2 * size and float(d.max()) < 0.5 * size, rid


def _attention(hidden, c, **more):
    from zedinfer_b200.parts import NormedAttentionMixer
    return NormedAttentionMixer(hidden, c["heads"], c["kv_heads"], c["dim"], v_head_dim=c["vdim"], scale=c["scale"], eps=1e-5, gate=True, **more)


def _left_mixer(hidden, c):
    from zedinfer_b200.config import PartSpec
    rot = c["rot"]
    return _attention(hidden, c, qk_norm="head", qkv_bias=True, out_bias=True, chunk=c["mask"]["size"],
                      position=PartSpec("rope_span", {"head_dim": c["dim"], "dims": rot["dims"], "theta": rot["base"], "interleaved": True,
                                                      "scaling": rot.get("scaling")}))


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("heads,kv,dim,vdim,chunk,dims,base,scaling,page", [
    (4, 2, 32, 16, 13, 16, 5000.0, (4.0, 1.0, 4.0, 64), 4), (2, 1, 64, 64, 40, 64, 10000.0, None, 16), (4, 4, 128, 128, 21, 32, 300.0, (2.0, 1.0, 3.0, 20), 16),
    (3, 3, 18, 26, 3, 2, 77.0, None, 8), (8, 2, 64, 128, 29, 24, 2e5, (8.0, 1.0, 4.0, 100), 16), (1, 1, 8, 8, 1, 8, 10.0, None, 8), (6, 3, 64, 64, 16, 64, 500.0, None, 16),
    (20, 1, 64, 64, 500, 32, 500.0, None, 32)])
def test_attention_in_chunks_with_normed_heads_and_a_gate(dtype, heads, kv, dim, vdim, chunk, dims, base, scaling, page):
    """Over portions and single tokens of two requests in shared steps, in a pool that gives the pages of a finished chunk to
    whoever asks next."""
    from zedinfer_b200.cache import CacheManager
    hidden = 80
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    c = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": 2.0 * dim ** -0.5, "mask": {"size": chunk}, "rot": rot}
    mixer = _left_mixer(hidden, c)
    t = bind_random(mixer, dtype, seed=dim + heads, scale=0.2, overrides={"q.norm": 1 + 0.3 * torch.randn(dim), "k.norm": 1 + 0.3 * torch.randn(dim)})
    cache = CacheManager([(0, mixer.cache_need())], page, max_requests=2)
    cache.allocate_device(40, dtype, DEV)
    g = torch.Generator().manual_seed(7)
    xs = {"a": torch.randn(61, hidden, generator=g).to(dtype), "b": torch.randn(19, hidden, generator=g).to(dtype)}
    got, = feed([mixer], [cache.view_for_call(0)], cache, dtype, xs, SCHEDULE_AB)
    for rid, x in xs.items():
        assert rel_err(got[rid], BP.chunked_attention(x.double(), t, "", c, 1e-5)) < tol_part(dtype, 2e-5, 3e-2), rid


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("heads,kv,dim,vdim,rows,farthest,heat,page", [
    (4, 2, 32, 16, 16, 40, (0.4, 16), 4), (2, 1, 64, 64, 32, 1000, None, 16), (4, 4, 128, 128, 10, 21, (0.3, 8), 16), (3, 3, 18, 26, 2, 5, (0.5, 1), 8),
    (8, 2, 64, 128, 8, 33.5, (0.1, 500), 16), (1, 1, 8, 8, 2, 2, (1.0, 2), 8), (36, 2, 64, 64, 24, 60, (0.2, 10), 16), (6, 3, 64, 64, 12, 50, None, 24)])
def test_attention_with_a_bias_by_distance_mixed_values_and_a_temperature(dtype, heads, kv, dim, vdim, rows, farthest, heat, page):
    """Two layers on the same input, the second mixing in the first one's values; large tables, so that a bucket or a head that is
    off shows; pages of 24 tokens take the kernels that gather rows one by one."""
    from zedinfer_b200.cache import CacheManager
    hidden = 80
    c = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": dim ** -0.5, "bias_max": farthest, "v_mix": True}
    if heat:
        c["q_temp"] = {"coef": heat[0], "every": heat[1]}
    mixers = [_attention(hidden, c, qk_norm="row", heat=heat, value_mix=mix, bias_rows=rows, bias_max=farthest) for mix in ("first", "mix")]
    ts = [bind_random(m, dtype, seed=dim + heads + i, scale=0.2, overrides={
        "rel": torch.randn(rows, heads) * 2, "vmix": torch.tensor(0.7 - i), "q.norm": 1 + 0.3 * torch.randn(heads * dim),
        "k.norm": 1 + 0.3 * torch.randn(kv * dim)}) for i, m in enumerate(mixers)]
    cache = CacheManager([(i, m.cache_need()) for i, m in enumerate(mixers)], page, max_requests=2)
    cache.allocate_device(40, dtype, DEV)
    g = torch.Generator().manual_seed(7)
    xs = {"a": torch.randn(61, hidden, generator=g).to(dtype), "b": torch.randn(19, hidden, generator=g).to(dtype)}
    got = feed(mixers, [cache.view_for_call(i) for i in range(2)], cache, dtype, xs, SCHEDULE_AB)
    tol = tol_part(dtype, 2e-5, 3e-2)
    for rid, x in xs.items():
        shared = {}
        refs = [BP.biased_attention(x.double(), t, "", c, 1e-5, shared) for t in ts]
        assert rel_err(got[0][rid], refs[0]) < tol and rel_err(got[1][rid], refs[1]) < tol, rid
        alone = BP.biased_attention(x.double(), ts[1], "", c, 1e-5, {})
        flat = BP.biased_attention(x.double(), dict(ts[0], rel=torch.zeros(rows, heads, dtype=F64)), "", c, 1e-5, {})
        if rid == "a":                                                     # the premise: either mechanism left out would show
            assert rel_err(alone, refs[1]) > 3 * tol and rel_err(flat, refs[0]) > 3 * tol
    with pytest.raises(RuntimeError):
        feed(mixers[1:], [cache.view_for_call(1)], cache, dtype, {"z": xs["b"]}, [["end:a", "end:b"], [("z", 3)]])


def _identity_tensors(dim, vdim, hidden, with_bias):
    """x = [query row | key row | value marks]: projections pick their own part; the gate is one half everywhere."""
    wq, wk, wv = torch.zeros(dim, hidden), torch.zeros(dim, hidden), torch.zeros(vdim, hidden)
    wq[:, :dim], wk[:, dim:2 * dim], wv[:, 2 * dim:] = torch.eye(dim), torch.eye(dim), torch.eye(vdim)
    t = {"q": wq, "k": wk, "v": wv, "o": 2.0 * torch.eye(hidden, vdim), "g": torch.zeros(vdim, hidden), "q.norm": torch.ones(dim), "k.norm": torch.ones(dim)}
    if with_bias:
        t.update({"q.b": torch.zeros(dim), "k.b": torch.zeros(dim), "v.b": torch.zeros(vdim), "o.b": torch.zeros(hidden)})
    return t


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("dim,vdim,chunk,page,dims,base", [(32, 24, 150, 16, 32, 50.0), (64, 128, 97, 8, 32, 300.0), (128, 128, 256, 16, 64, 1000.0), (16, 24, 590, 4, 16, 20.0),
                                                           (64, 64, 128, 16, 64, 2e5), (64, 64, 80, 24, 32, 100.0)])
def test_one_key_answers_just_inside_a_chunk_and_none_just_outside(dtype, dim, vdim, chunk, page, dims, base):
    """One head, 640 tokens.  A query aligned with the first key of its own chunk gets that key's value; one aligned with the key
    just before its chunk does not.  The chunk's own first token sees itself alone.  Asked from inside a prompt's portion and
    by tokens fed alone, with portions cut off the chunks' and the pages' edges."""
    from zedinfer_b200.cache import CacheManager
    total = 640
    hidden = 2 * dim + vdim
    c = {"heads": 1, "kv_heads": 1, "dim": dim, "vdim": vdim, "scale": 200.0 / dim, "mask": {"size": chunk}, "rot": {"base": base, "dims": dims}}
    mixer = _left_mixer(hidden, c)
    tensors = _identity_tensors(dim, vdim, hidden, True)
    mixer.bind({k: v.to(dtype).to(DEV) for k, v in tensors.items()})
    last = (total - 1) // chunk * chunk                                     # the last chunk's first token
    inside = {total - 1: last, total - 3: last}                             # decoded
    outside = {total - 2: last - 1, total - 4: last - 1}
    if last > 2 * chunk:                                                    # in a prompt's portion too
        inside.update({last - 1: last - chunk, last - chunk + 1: last - chunk})
        outside.update({last: last - 1, last - 2: last - chunk - 1})
    raw = torch.zeros(dim, dtype=F64)
    raw[0:dims:2] = 1.0
    keys, queries = torch.zeros(total, dim, dtype=F64), torch.zeros(total, dim, dtype=F64)
    for p, j in {**inside, **outside}.items():
        keys[j] = raw
        queries[p] = BP.turn_pairs(raw[None, None], torch.tensor([j - p]), dims, base)[0, 0]
    marks = torch.randn(total, vdim, generator=torch.Generator().manual_seed(dim)).double()
    x = torch.cat([queries, keys, marks], dim=1).to(dtype)
    cache = CacheManager([(0, mixer.cache_need())], page, max_requests=1)
    cache.allocate_device(total // page + 2, dtype, DEV)
    schedule = [[("r", 201)], [("r", 2)], [("r", total - 208)]] + [[("r", 1)]] * 5
    got = feed([mixer], [cache.view_for_call(0)], cache, dtype, {"r": x}, schedule, table_width=170)[0]["r"]
    ref = BP.chunked_attention(x.double(), {k: v.double() for k, v in tensors.items()}, "", c, 1e-5)
    assert rel_err(got, ref) < (1e-3 if dtype == torch.float32 else 3e-2)
    vals = x.double()[:, 2 * dim:]
    for p, j in inside.items():
        assert rel_err(ref[p, :vdim], vals[j]) < 3e-2, (p, j)                  # the premise: that key alone answers
    for p, j in outside.items():
        assert float((ref[p, :vdim] - vals[j]).abs().max()) > 0.5, (p, j)      # the premise: it does not


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("dim,vdim,rows,farthest,page", [(32, 24, 14, 250, 16), (64, 64, 32, 700, 16), (128, 128, 10, 130, 16), (64, 64, 6, 90, 24), (16, 8, 12, 2000, 4)])
@pytest.mark.parametrize("bucket", ["zero", "half", "inner", "last"])
def test_a_bucket_that_stands_out_answers_from_its_first_distance_to_its_last(dtype, dim, vdim, rows, farthest, page, bucket):
    """Scores all zero but for one bucket's large number: a query gets the mean of exactly the values whose distance lies in that
    bucket, so that one distance more or less shows, in prompts and in decoding; and one key that stands out among hundreds
    although the bias is against it."""
    from zedinfer_b200.cache import CacheManager
    total, hidden = 640, 2 * dim + vdim
    b = {"zero": 0, "half": rows // 2, "inner": rows - 2, "last": rows - 1}[bucket]
    c = {"heads": 1, "kv_heads": 1, "dim": dim, "vdim": vdim, "scale": 200.0 / dim, "bias_max": farthest}
    mixer = _attention(hidden, c, qk_norm="row", bias_rows=rows, bias_max=farthest)
    rel = torch.zeros(rows, 1)
    rel[b] = 30.0
    tensors = dict(_identity_tensors(dim, vdim, hidden, False), rel=rel)
    mixer.bind({k: v.to(dtype).to(DEV) for k, v in tensors.items()})
    keys, queries = torch.zeros(total, dim), torch.zeros(total, dim)
    keys[17], keys[311] = torch.eye(dim)[0], torch.eye(dim)[1]
    far = {639: 17, 500: 17, 636: 311, 312: 311}
    for p, j in far.items():
        queries[p] = keys[j]
    # a slope beside the noise: a set of values that is off by one has another mean
    marks = torch.randn(total, vdim, generator=torch.Generator().manual_seed(dim)) + torch.arange(total)[:, None] / 64.0
    x = torch.cat([queries, keys, marks], dim=1).to(dtype)
    cache = CacheManager([(0, mixer.cache_need())], page, max_requests=1)
    cache.allocate_device(total // page + 2, dtype, DEV)
    schedule = [[("r", 299)], [("r", 2)], [("r", total - 309)]] + [[("r", 1)]] * 8
    got = feed([mixer], [cache.view_for_call(0)], cache, dtype, {"r": x}, schedule, table_width=170)[0]["r"]
    ref = BP.biased_attention(x.double(), {k: v.double() for k, v in tensors.items()}, "", c, 1e-5, {})
    scale = float(ref[:, :vdim].abs().max())
    err = (got.double() - ref)[:, :vdim].abs().max(dim=1).values
    assert float(err.max()) < (1e-4 if dtype == torch.float32 else 2e-2) * scale
    vals = x.double()[:, 2 * dim:]
    for p, j in far.items():
        assert rel_err(ref[p, :vdim], vals[j]) < 1e-2                      # the premise: that key alone answers


# ---------------------------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("bogivik_models")
    return {name: BT.make_model_dir(root, name) for name in BT.CONFIGS}


def make_requests(cfg, lengths, seed):
    rng = random.Random(seed)
    return {f"r{i}": [rng.randrange(cfg["vocab"]) for _ in range(n)] for i, n in enumerate(lengths)}


_plain_cache = {}


def expected_logits(model_dir, requests):
    if model_dir not in _plain_cache:
        _plain_cache[model_dir] = BP.read_model(model_dir, F64)
    cfg, w = _plain_cache[model_dir]
    return {rid: BP.forward(cfg, w, toks).float() for rid, toks in requests.items()}


def judge(got, exp, dtype):
    """float32: every position within the tolerance.  bfloat16: rounding errors have a tail, the same however the work is
    cut: at most 2 % of the positions may be beyond the tolerance, none beyond four times it."""
    tol = tol_for(dtype)
    errs = {key: float((row - exp[key[0]][key[1]]).abs().max()) / max(1.0, float(exp[key[0]].abs().max()))
            for key, row in got.items()}
    over = sorted((k for k, e in errs.items() if not e <= tol), key=lambda k: (str(k[0]), k[1]))
    allowed = 0 if dtype == "float32" else max(1, len(errs) // 50)
    assert len(over) <= allowed, f"{len(over)} of {len(errs)} positions beyond {tol}; first {over[0]} with {errs[over[0]]}"
    assert all(e <= 4 * tol for e in errs.values()), max(errs.values())


LENGTHS = {"A": [7, 13, 95, 45], "B": [1, 17, 150, 64], "C": [110, 5, 60], "D": [50, 2, 61], "E": [40, 3, 90], "F": [33, 1, 70]}
PAGES = {"A": 4, "B": 16, "C": 8, "D": 8, "E": 16, "F": 8}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D", "E", "F"])
@pytest.mark.parametrize("family", ["whole", "tail", "chunks", "mixed"])
def test_cuts_match_plain(models, name, dtype, family):
    """Whole prompts; a tail decoded token by token; portions down to two tokens; mixed batches of unequal requests in a
    pool so small that pages and state slots are handed out again."""
    from zedinfer_b200.engine.core import EngineCore
    cfg, _ = BT.CONFIGS[name]
    requests = make_requests(cfg, LENGTHS[name] + ([64, 31, 77] if family == "mixed" else []), seed=5)
    if family == "tail":
        steps = traces.tail_decode(requests, tail=40)
    else:
        steps = {"whole": traces.whole, "chunks": traces.chunks, "mixed": traces.mixed}[family](requests)
    page = PAGES[name]
    need = traces.max_live_tokens(steps, round_to=page)
    core = EngineCore(models[name], dtype, page_size=page, num_pages=max(1, need // page), max_requests=4)
    got = run_trace(core, steps)
    core.check_kernels()
    judge(got, expected_logits(models[name], requests), dtype)
    assert core.cache.num_live == 0 and all(g.pool.num_used == 0 for g in core.cache.groups)
    assert core.cache.slots.num_free_slots == core.cache.slots.num_slots


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("B", "float32"), ("B", "bfloat16"), ("C", "bfloat16"), ("D", "bfloat16")])
def test_many_decoding_requests_with_and_without_graphs(models, name, dtype, graphs):
    """Steps as a scheduler makes them: up to 12 decoding requests beside one prompt portion, then decode-only steps whose
    number of rows falls to one; with graphs the decode-only steps replay captured buckets whose rows of padding hold no
    state slot."""
    from zedinfer_b200.engine.core import EngineCore
    cfg, _ = BT.CONFIGS[name]
    rng = random.Random(8)
    requests = make_requests(cfg, [rng.randint(40, 90) for _ in range(15)], seed=3)
    steps = traces.decode_heavy(requests, seed=4, max_live=12, tail=(8, 30), portion=32)
    need = traces.max_live_tokens(steps, round_to=16)
    core = EngineCore(models[name], dtype, page_size=16, num_pages=need // 16, max_requests=16, cuda_graphs=graphs)
    core.GPU_BOUND_RATIO = float("inf")
    assert core.capture_safe, core.capture_blockers
    got = run_trace(core, steps)
    core.check_kernels()
    judge(got, expected_logits(models[name], requests), dtype)
    if graphs:
        assert core._decode_graphs
    assert core.cache.num_live == 0 and all(g.pool.num_used == 0 for g in core.cache.groups)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_and_the_first_tokens(models, dtype):
    """One token, two tokens, and a request decoded for 260 steps from a prompt of three: every chunk opens over decoded tokens many
    times, the distances run past the last bucket, the matrix memory goes through hundreds of single-token steps."""
    from zedinfer_b200.engine.core import EngineCore
    cfg, _ = BT.CONFIGS["A"]
    requests = make_requests(cfg, [1, 2, 263], seed=9)
    steps = traces.tail_decode(requests, tail=260)
    core = EngineCore(models["A"], dtype, page_size=4, num_pages=80, max_requests=2)
    judge(run_trace(core, steps), expected_logits(models["A"], requests), dtype)


@pytest.mark.parametrize("name", ["A", "C", "D", "F"])
def test_float32_is_the_same_however_it_is_cut(models, name):
    """The same positions through four different schedules: the same bits (every float32 sum of the design has one order,
    which depends on constants alone; the recurrence runs token by token whatever the portions)."""
    from zedinfer_b200.engine.core import EngineCore
    cfg, _ = BT.CONFIGS[name]
    requests = make_requests(cfg, [90, 41], seed=2)
    runs = []
    for steps in (traces.whole(requests), traces.tail_decode(requests, tail=20), traces.chunks(requests), traces.mixed(requests)):
        core = EngineCore(models[name], "float32", page_size=16, num_pages=40, max_requests=4)
        runs.append(run_trace(core, steps))
    for other in runs[1:]:
        assert all(torch.equal(other[k], runs[0][k]) for k in runs[0])


@pytest.mark.parametrize("name,graphs", [("A", False), ("A", True), ("B", True), ("C", False), ("D", True), ("F", True)])
def test_greedy_generation_equals_plain(models, name, graphs):
    """Through the Python entry point and its scheduler: prompts in portions of five, a pool of pages (of layers with chunks only
    as large as they need) and three state slots that the requests fill again, greedy tokens equal to the plain
    implementation's."""
    from zedinfer_b200 import GenerationConfig, SchedulerConfig
    from zedinfer_b200.engine import InferenceEngine
    cfg, _ = BT.CONFIGS[name]
    rng = random.Random(4)
    prompts = [[rng.randrange(cfg["vocab"]) for _ in range(n)] for n in (9, 23, 1, 14, 6)]
    engine = InferenceEngine.create(models[name], SchedulerConfig(num_kv_pages=30, kv_block_size=4, max_batch_requests=3,
                                                                  max_prefill_tokens=5, cuda_graphs=graphs),
                                    dtype="float32")
    results = engine.generate_batch(prompts, GenerationConfig(max_new_tokens=20, ignore_eos=True))
    pcfg, w = BP.read_model(models[name], F64)
    for p, r in zip(prompts, results):
        assert r.finish_reason == "length"
        assert r.output_ids == BP.greedy(pcfg, w, p, 20)
    st = engine.cache_stats()
    assert st["live_requests"] == 0 and st["free_pages"] == st["pages_per_group"]


@pytest.mark.parametrize("name,dtype", [("B", "bfloat16"), ("B", "float32"), ("D", "float32"), ("E", "bfloat16")])
def test_trace_program_on_a_bogivik_folder(models, tmp_path, name, dtype):
    """The program on a folder with both kinds of layer, on one without a state slot and on one without layers over every key."""
    cfg, _ = BT.CONFIGS[name]
    requests = make_requests(cfg, [70, 9, 33, 50, 21], seed=6)
    steps = traces.mixed(requests, seed=1)
    need = traces.max_live_tokens(steps, round_to=64)
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", models[name], "--dtype", dtype,
                           "--out", str(out), "--max-tokens", str(need)],
                          input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done ")] == [f"done {i}" for i in range(len(steps))]
    got, progress = {}, {}
    for st in steps:
        rows = np.fromfile(out / f"{st['step']}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
        row = 0
        for e in st["entries"]:
            base = progress.get(e["id"], 0)
            for j in e["want"]:
                got[(e["id"], base + j)] = torch.from_numpy(rows[row].copy())
                row += 1
            progress[e["id"]] = base + len(e["tokens"])
        assert row == rows.shape[0]
    judge(got, expected_logits(models[name], requests), dtype)


def test_command_line_programs_take_the_design(tmp_path, capsys):
    """From a bare config.json with weights drawn on the device: the bench program, continuous batching, and the
    consistency program, which returns 0 only if every float32 logit is the same bit pattern however the work is cut."""
    from zedinfer_b200.cli import batch_bench, bench, consistency
    path = tmp_path / "config.json"
    path.write_text(json.dumps(BT.BG_A))
    common = [str(path), "--random-weights", "7", "--kv-pages", "40", "--max-seq-len", "128"]
    assert bench.main(common + ["-p", "24", "-d", "5", "-r", "1"]) == 0
    out = capsys.readouterr().out
    assert "Prefill:" in out and "Decode :" in out
    assert batch_bench.main(common + ["-b", "5", "-p", "6", "--prefill-len-max", "40", "-d", "7", "-r", "1",
                                      "--warmup-rounds", "1", "--max-prefill-tokens", "16"]) == 0
    assert "5 requests, 35 tokens generated" in capsys.readouterr().out
    assert consistency.main([str(path), "--random-weights", "5", "--tokens", "120", "--requests", "5"]) == 0
    lines = [json.loads(l) for l in capsys.readouterr().out.strip().splitlines()]
    assert all(l["values_not_bit_equal"] == 0 for l in lines if l["dtype"] == "float32")
