"""The Fedutar design on the GPU against the plain restatement in oracle/fedutar_oracle.py.

Every test builds its own small configuration and random weights (none of them a published model's sizes).  Logits are
compared at EVERY position.  The exact engine computes in fp32 on the bf16 weights, so its bound is rounding: 1e-4 of the
largest logit.  The serving form keeps the attention's queries, keys, values and softmax weights and the retention's projections
in bf16, which bounds the agreement there.
"""
import copy
import json
import os
import subprocess

import numpy as np
import pytest
import torch

from oracle import fedutar_oracle as O

pytestmark = pytest.mark.gpu
TOL = 1e-4
TOL16 = 2e-2


# ------------------------------------------------------------------------------------------------ configurations
def decays(n, lo=2, hi=8):
    return [1.0 - 2.0 ** -(lo + (hi - lo) * h / max(1, n - 1)) for h in range(n)]


def parallel(heads=4, kv_heads=2, dim=20, vdim=12, scale=0.3, temp=(0.25, 16), rheads=3, rdim=16, rvdim=24, rot=12, base=900.0, ls=0.7, rs=1.2,
             decay=None):
    left = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "vdim": vdim}
    if temp:
        left["q_temp"] = {"coef": temp[0], "every": temp[1]}
    right = {"decay": decay or decays(rheads), "dim": rdim, "heads": rheads, "vdim": rvdim}
    if rot:
        right["rot"] = {"base": base, "dims": rot}
    return {"type": "parallel", "mixer": {"left": left, "left_scale": ls, "right": right, "right_scale": rs}}


def moe(ff=24, experts=6, top=2, limit=1.25):
    return {"expert": {"ff": ff, "limit": limit}, "kind": "moe", "router": {"experts": experts, "top": top}}


def dense(ff=44):
    return {"ff": ff, "kind": "dense"}


def layer(mixer, mlp=None):
    return {**copy.deepcopy(mixer), "mlp": mlp}


def make(layers, width=80, vocab=150, eps=1e-5, seed=0, embed_scale=3.0, logit_scale=0.2, softcap=8.0, loop=None, tweak=None):
    from fasttalk_llm_microservice_b200.layered import init_weights, spec_from_config, tensor_shapes
    cfg = {"architecture": "Fedutar", "embedding": {"scale": embed_scale}, "layers": copy.deepcopy(layers), "logit_scale": logit_scale,
           "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if softcap:
        cfg["logit_softcap"] = softcap
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    spec = spec_from_config(cfg, None, name="test")
    assert spec.config() == cfg
    assert spec_from_config(spec.config(), tensor_shapes(spec), name="test") == spec
    w = init_weights(spec, seed=seed)
    if tweak:
        tweak(w)
    return spec, w


def engine(spec, w, **kw):
    from fasttalk_llm_microservice_b200 import build
    from fasttalk_llm_microservice_b200.engine import Engine, EngineLimits
    build.build()
    lim = EngineLimits(**{"max_batch": 4, "max_batched_tokens": 512, "max_context": 512, "num_pages": 16,
                          "max_sessions": 4, "debug_logit_rows": 512, "exact_f32": True, **kw})
    return Engine(spec, w, lim, eos_ids=())


def oracle_logits(spec, w, tokens, cfg=None):
    with torch.no_grad():
        return O.forward(cfg or spec.config(), w, list(tokens)).numpy()


def rel(got, ref):
    return float(np.abs(got - ref).max() / np.abs(ref).max())


def tokens_of(spec, n, seed):
    return np.random.default_rng(seed).integers(0, spec.vocab, n).tolist()


def feed_cut(eng, sid, toks, cuts):
    """Feed `toks` to session `sid` in portions of the given sizes (the last size repeats); logits of every position."""
    out, pos, k = [], 0, 0
    while pos < len(toks):
        n = min(cuts[min(k, len(cuts) - 1)], len(toks) - pos)
        out.append(eng.feed([(sid, toks[pos:pos + n], list(range(n)))]))
        pos, k = pos + n, k + 1
    return np.concatenate(out)


def run_plan(eng, seqs, plan):
    """Feed the steps of `plan` ({session: tokens}) to the end of every sequence; logits of every position by session."""
    at, got = {n: 0 for n in seqs}, {n: [] for n in seqs}
    for step in plan:
        counts = {n: min(c, len(seqs[n]) - at[n]) for n, c in step.items()}
        counts = {n: c for n, c in counts.items() if c}
        if not counts:
            continue
        out, o = eng.feed([(n, seqs[n][at[n]:at[n] + c], list(range(c))) for n, c in counts.items()]), 0
        for n, c in counts.items():
            got[n].append(out[o:o + c])
            o, at[n] = o + c, at[n] + c
    assert all(at[n] == len(seqs[n]) for n in seqs)
    return {n: np.concatenate(g) for n, g in got.items()}


def sharpen(f):
    """Query gains `f` times larger: the softmax rests on a few keys, a lost or misplaced one shows."""
    def tweak(w):
        for k in list(w):
            if k.endswith("left.q.norm"):
                w[k] = (w[k].float() * f).to(torch.bfloat16)
    return tweak


MIXED = [layer(parallel(), dense()), layer(parallel(heads=6, kv_heads=3, dim=13, vdim=10, temp=None, rheads=2, rdim=10, rvdim=9, rot=4), moe()),
         layer(parallel(heads=3, kv_heads=1, dim=32, vdim=7, rheads=5, rdim=8, rvdim=16, rot=0, ls=1.0, rs=1.0)),
         layer(parallel(heads=2, kv_heads=2, temp=(0.5, 7), rheads=1, rdim=30, rvdim=5, rot=30, base=1e5), moe(ff=17, experts=4, top=1, limit=3.0))]
LOOP = (1, 3, 2)


# ------------------------------------------------------------------------------------------------ every mechanism alone
@pytest.mark.parametrize("layers,loop", [
    ([layer(parallel())], None),
    ([layer(parallel(rs=0.0))], None),
    ([layer(parallel(ls=0.0))], None),
    ([layer(parallel(rs=0.0, temp=None, heads=3, kv_heads=3))], None),
    ([layer(parallel(rs=0.0, heads=12, kv_heads=1, dim=7, vdim=70, temp=(1.5, 1)))], None),
    ([layer(parallel(heads=1, kv_heads=1, dim=1, vdim=1, rheads=1, rdim=2, rvdim=1, rot=2))], None),
    ([layer(parallel(heads=2, kv_heads=1, dim=140, vdim=200, rheads=2, rdim=150, rvdim=300, rot=100))], None),
    ([layer(parallel(ls=0.0, rot=0, rdim=33, rvdim=17))], None),
    ([layer(parallel(ls=0.0, rheads=4, decay=[1.0, 0.0, 0.5, 0.999]))], None),
    ([layer(parallel(), dense())], None),
    ([layer(parallel(), dense(ff=7))], None),
    ([layer(parallel(), moe())], None),
    ([layer(parallel(), moe(ff=7, experts=3, top=3, limit=0.1))], None),
    ([layer(parallel(), moe(ff=20, experts=40, top=1, limit=30.0))], None),
    ([layer(parallel()), layer(parallel())], (0, 1, 1)),
    ([layer(parallel()), layer(parallel(), dense())], (0, 2, 3)),
    ([layer(parallel()), layer(parallel(), moe()), layer(parallel(heads=2))], (1, 2, 4)),
    ([layer(parallel(), dense()), layer(parallel())], (1, 2, 2)),
    (MIXED, None),
    (MIXED, LOOP),
], ids=["both", "attention", "retention", "attention-plain", "attention-one-key-head", "tiny", "wide", "retention-unrotated", "decays", "dense",
        "dense-odd", "experts", "experts-all", "experts-many", "one-pass", "loop-all", "loop-middle", "loop-end", "mixed", "mixed-loop"])
def test_whole_prompt_matches_oracle(layers, loop):
    spec, w = make(layers, seed=3, loop=loop)
    eng = engine(spec, w)
    try:
        toks = tokens_of(spec, 150, 1)
        got = eng.feed([("s", toks, list(range(len(toks))))])
        assert rel(got, oracle_logits(spec, w, toks)) < TOL
    finally:
        eng.close()


@pytest.mark.parametrize("width,vocab,scale,lscale,cap,eps", [(70, 333, 1.0, 1.0, 0.0, 1e-6), (33, 50, 9.0, 0.05, 2.0, 1e-3),
                                                              (132, 128, 0.5, 0.7, 50.0, 1e-5)])
def test_other_sizes_and_constants(width, vocab, scale, lscale, cap, eps):
    spec, w = make(MIXED, width=width, vocab=vocab, embed_scale=scale, logit_scale=lscale, softcap=cap, eps=eps, loop=(0, 2, 3), seed=9)
    eng = engine(spec, w)
    try:
        toks = tokens_of(spec, 90, 2)
        ref = oracle_logits(spec, w, toks)
        assert rel(eng.feed([("s", toks, list(range(len(toks))))]), ref) < TOL
        assert rel(feed_cut(eng, "c", toks, [1, 2, 1, 7, 1]), ref) < TOL
    finally:
        eng.close()


def test_residual_after_every_layer_run():
    """The stream after every run of every layer, before the projection ahead of the next pass."""
    spec, w = make(MIXED, seed=4, loop=(0, 3, 3))
    eng = engine(spec, w)
    try:
        toks = tokens_of(spec, 70, 5)
        eng.debug_trail(True)
        eng.feed([("s", toks, [])])
        got = eng.read_trail(len(toks))
        trail = []
        with torch.no_grad():
            O.forward(spec.config(), w, toks, trail=trail)
        assert len(trail) == got.shape[0] == 10
        for i, t in enumerate(trail):
            assert rel(got[i], t.numpy()) < TOL, i
    finally:
        eng.close()


def test_every_part_of_the_design_matters():
    """Leaving out or changing one part moves the logits by far more than the bound, so the agreement with the restatement says that
    each of them is computed."""
    spec, w = make(MIXED, seed=5, loop=LOOP)
    eng = engine(spec, w)
    try:
        toks = tokens_of(spec, 160, 6)
        ref = oracle_logits(spec, w, toks)
        assert rel(feed_cut(eng, "a", toks, [100, 1, 1, 1, 50, 1]), ref) < TOL
    finally:
        eng.close()
    for name, value in {"l0.mix.left.q.norm": 1.0, "l0.mix.left.k.norm": 1.0, "l0.mix.left.g": 0.0, "l1.mix.right.g": 0.5, "l0.mlp.gate.b": 0.0,
                        "l0.mlp.up.b": 0.0, "l0.mlp.down.b": 0.0, "l0.norm1b": 1.0, "l1.norm2b": 1.0, "l2.norm1": 1.0, "final.norm": 1.0}.items():
        w2 = dict(w)
        w2[name] = torch.full_like(w[name], value)
        assert rel(oracle_logits(spec, w2, toks), ref) > 20 * TOL, name
    w2 = dict(w)
    w2["loop.in"] = w["loop.in"].clone()
    w2["loop.in"][:, spec.width:] = 0                   # a pass reads the embedding output too
    assert rel(oracle_logits(spec, w2, toks), ref) > 20 * TOL
    for path, value in ((("logit_scale",), 0.21), (("logit_softcap",), 8.5), (("embedding", "scale"), 2.0), (("loop", "times"), 1),
                        (("loop", "start"), 2), (("layers", 0, "mixer", "left", "q_temp", "coef"), 0.3),
                        (("layers", 0, "mixer", "left", "q_temp", "every"), 15), (("layers", 0, "mixer", "left", "scale"), 0.4),
                        (("layers", 0, "mixer", "right", "rot", "base"), 300.0), (("layers", 0, "mixer", "right", "rot", "dims"), 10),
                        (("layers", 0, "mixer", "right", "decay"), [0.7, 0.9, 0.99]), (("layers", 0, "mixer", "left_scale"), 0.8),
                        (("layers", 1, "mlp", "expert", "limit"), 1.0)):
        cfg = spec.config()
        d = cfg
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        assert rel(oracle_logits(spec, w, toks, cfg), ref) > 20 * TOL, path


# ------------------------------------------------------------------------------------------------ portions, decoding
@pytest.mark.parametrize("exact", [True, False], ids=["exact-fp32", "tensor-cores"])
@pytest.mark.parametrize("cuts", [[1], [2], [3, 2, 29, 1, 1, 17, 2], [64], [63, 1, 1, 64, 2], [65, 2], [129, 40, 2]],
                         ids=["token-by-token", "twos", "ragged", "pages", "around-pages", "over-a-page", "over-a-run"])
def test_portions_and_decoding_match_the_whole_prompt(cuts, exact):
    # every expert chosen: bf16 attention must not meet a close choice
    layers = [dict(l, mlp=dict(l["mlp"], router={"experts": 3, "top": 3})) if (l["mlp"] or {}).get("kind") == "moe" else l for l in MIXED]
    spec, w = make(MIXED if exact else layers, seed=7, loop=LOOP)
    eng = engine(spec, w, exact_f32=exact)
    try:
        toks = tokens_of(spec, 200, 8)
        ref = oracle_logits(spec, w, toks)
        whole = eng.feed([("w", toks, list(range(len(toks))))])
        got = feed_cut(eng, "c", toks, cuts)
        tol = TOL if exact else TOL16
        assert rel(whole, ref) < tol and rel(got, ref) < tol
        assert rel(got, whole) < (2e-5 if exact else TOL16)
    finally:
        eng.close()


def test_first_tokens_and_long_decoding():
    spec, w = make(MIXED, seed=19, loop=LOOP)
    eng = engine(spec, w)
    try:
        toks = tokens_of(spec, 300, 21)
        ref = oracle_logits(spec, w, toks)
        got = feed_cut(eng, "a", toks, [1, 1, 1, 2, 1, 30, 1])      # a sequence that starts with single tokens, then 264 decoded
        assert rel(got[:8], ref[:8]) < TOL
        assert rel(got, ref) < TOL
    finally:
        eng.close()


def only(side, w):
    """Leave one side of the first layer's mixer: the other side's output projection is zero."""
    w[f"l0.mix.{side}.o"][:] = 0


@pytest.mark.parametrize("exact", [True, False], ids=["exact-fp32", "tensor-cores"])
@pytest.mark.parametrize("kv_heads,dim,vdim", [(1, 16, 24), (4, 96, 40)])
def test_one_far_key_among_hundreds(kv_heads, dim, vdim, exact):
    """Token 0 lives on coordinate 0 of the stream, token 1 on coordinate 1.  Every query points along channel 0, which only token
    1's key meets: one marked token in a sequence of equal tokens takes most of the weight for everyone after it, however far, and
    none before it; at and around page borders, in a prompt, in portions and in decoding."""
    def tweak(w):
        for n in ("embed", "l0.mix.left.q", "l0.mix.left.k"):
            w[n][:] = 0
        w["embed"][0, 0] = w["embed"][1, 1] = 1.0
        for h in range(4):
            w["l0.mix.left.q"][h * dim, 0] = w["l0.mix.left.q"][h * dim, 1] = 1.0
        for g in range(kv_heads):
            w["l0.mix.left.k"][g * dim, 1] = 1.0
        for n in ("l0.norm1", "l0.mix.left.q.norm", "l0.mix.left.k.norm"):
            w[n][:] = 1.0
        only("right", w)
    spec, w = make([layer(parallel(heads=4, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=9.0 / dim, temp=None))], width=64, vocab=40, seed=2,
                   embed_scale=1.0, tweak=tweak)
    eng = engine(spec, w, max_batched_tokens=704, max_context=704, debug_logit_rows=704, exact_f32=exact)
    try:
        n = 700
        plain = oracle_logits(spec, w, [0] * n)
        for mark in (0, 63, 64, 130, 319):
            toks = [0] * n
            toks[mark] = 1
            ref = oracle_logits(spec, w, toks)
            seen = np.abs(ref - plain).max(-1) / np.abs(ref).max()
            assert seen[mark:].min() > 5e-2 and (mark == 0 or seen[:mark].max() < 1e-9)
            for cuts in ([n], [mark + 1, 1, 1, 62, 1, 150, 1, 1, 300, 1], [64, 2, 2]):
                got = feed_cut(eng, "s", toks, cuts)
                eng.close_session("s")
                assert rel(got, ref) < (TOL if exact else TOL16), (mark, cuts)
    finally:
        eng.close()


@pytest.mark.parametrize("exact", [True, False], ids=["exact-fp32", "tensor-cores"])
def test_a_far_write_stays_in_the_state(exact):
    """Retention alone, decays 1 and close to 1, no rotation: the first token is still felt hundreds of tokens later, through run
    borders, portions and single tokens; a state that was lost or started over would show."""
    layers = [layer(parallel(rheads=3, rdim=32, rvdim=32, rot=0, decay=[1.0, 0.9999, 0.99]))]
    spec, w = make(layers, width=64, vocab=50, seed=8, tweak=lambda w: only("left", w))
    eng = engine(spec, w, max_batched_tokens=704, max_context=704, debug_logit_rows=704, exact_f32=exact)
    try:
        toks = [7] + [int(t) for t in np.random.default_rng(3).integers(0, 5, 639)]
        ref = oracle_logits(spec, w, toks)
        lost = oracle_logits(spec, w, [3] + toks[1:])
        assert rel(lost[400:], ref[400:]) > 2 * TOL
        tol = TOL if exact else TOL16
        for cuts in ([640], [1, 127, 1, 128, 1, 129, 2, 1], [300, 1, 1, 64, 2, 192, 1]):
            assert rel(feed_cut(eng, "s", toks, cuts), ref) < tol, cuts
            eng.close_session("s")
    finally:
        eng.close()


@pytest.mark.parametrize("exact", [True, False], ids=["exact-fp32", "tensor-cores"])
def test_steps_of_the_temperature(exact):
    """Sharpened queries with a large coefficient: a temperature that steps one position early or late is far outside the bound."""
    def at(every):
        return make([layer(parallel(temp=(2.0, every), dim=32, vdim=32, heads=4, kv_heads=2))], seed=6,
                    tweak=lambda w: (sharpen(2.0)(w), only("right", w)))
    spec, w = at(40)
    eng = engine(spec, w, exact_f32=exact)
    try:
        toks = tokens_of(spec, 130, 4)
        ref = oracle_logits(spec, w, toks)
        tol = TOL if exact else TOL16
        got = feed_cut(eng, "a", toks, [37, 1, 1, 1, 1, 38, 1, 1, 40, 1])
        assert rel(got, ref) < tol and rel(eng.feed([("b", toks, list(range(130)))]), ref) < tol
    finally:
        eng.close()
    late = oracle_logits(*at(41), toks)                     # steps at p = 40 and 81 instead of 39 and 79
    assert rel(late[39:40], ref[39:40]) > 2 * TOL16 and rel(late[79:81], ref[79:81]) > TOL16 and rel(late[:39], ref[:39]) < 1e-9


# ------------------------------------------------------------------------------------------------ batches, pools
def test_unequal_requests_in_one_batch_match_each_alone():
    spec, w = make(MIXED, seed=13, loop=LOOP)
    eng = engine(spec, w)
    try:
        seqs = {n: tokens_of(spec, ln, 20 + i) for i, (n, ln) in enumerate([("a", 140), ("b", 33), ("c", 70), ("d", 9)])}
        ref = {n: oracle_logits(spec, w, t) for n, t in seqs.items()}
        alone = {}
        for n, t in seqs.items():
            alone[n] = eng.feed([(n + "-alone", t, list(range(len(t))))])
            eng.close_session(n + "-alone")
        # a schedule of mixed steps: portions of some beside single tokens of others, one request pausing for a step
        plan = [{"a": 64, "b": 1}, {"a": 2, "b": 1, "c": 29}, {"b": 16, "c": 1, "d": 3}, {"a": 1, "c": 1, "d": 1},
                {"a": 70, "b": 15, "c": 39, "d": 5}, {"a": 3}]
        got = run_plan(eng, seqs, plan)
        for n in seqs:
            assert rel(got[n], ref[n]) < TOL, n
            assert rel(got[n], alone[n]) < 2e-5, n
    finally:
        eng.close()


@pytest.mark.parametrize("exact", [True, False], ids=["exact-fp32", "tensor-cores"])
def test_pages_and_slots_are_used_again(exact):
    """A pool of 6 pages and 2 slots serves six sequences, one after the other and two at a time: what an ended session left in its
    pages and states (of every layer run) must not reach the next one."""
    layers = [layer(parallel(heads=2, kv_heads=1, dim=16, vdim=16, scale=1.0, rdim=32, rvdim=32, decay=[1.0, 0.999, 0.9]), moe(experts=3, top=3)),
              layer(parallel(heads=3, kv_heads=3, dim=64, vdim=32), dense())]
    spec, w = make(layers, seed=17, loop=(0, 1, 3))
    tol = TOL if exact else TOL16
    eng = engine(spec, w, max_batch=2, max_sessions=2, num_pages=6, max_context=384, max_batched_tokens=384, debug_logit_rows=384,
                 exact_f32=exact)
    try:
        seqs = [tokens_of(spec, ln, 40 + i) for i, ln in enumerate([190, 100, 130, 64, 65, 180])]
        ref = [oracle_logits(spec, w, t) for t in seqs]
        for i in (0, 1):                                       # alone, the whole pool in turn
            assert rel(feed_cut(eng, f"s{i}", seqs[i], [50, 1, 1, 90]), ref[i]) < tol
            eng.close_session(f"s{i}")
            assert eng.stats()["free_pages"] == 6
        for a, b in ((2, 3), (4, 5)):                          # two at a time
            got = run_plan(eng, {f"s{a}": seqs[a], f"s{b}": seqs[b]},
                           [{f"s{a}": 37, f"s{b}": 20 if k == 0 else 1 + 34 * (k % 2)} for k in range(14)])
            for i in (a, b):
                assert rel(got[f"s{i}"], ref[i]) < tol
                eng.close_session(f"s{i}")
        for first in (1, 2, 40):                               # a fresh sequence in a used slot, begun with one, a few or many tokens
            assert rel(feed_cut(eng, "again", seqs[2], [first, 1, 2, 40, 1]), ref[2]) < tol
            eng.close_session("again")
        st = eng.stats()
        assert st["free_pages"] == 6 and st["live_sessions"] == 0
    finally:
        eng.close()


# ------------------------------------------------------------------------------------------------ tensor cores
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 4, 32, 32), (10, 2, 96, 160), (8, 2, 128, 128), (5, 1, 20, 33), (16, 1, 64, 64), (40, 2, 16, 8),
                                                     (2, 2, 200, 100), (4, 2, 256, 256), (3, 3, 64, 300), (2, 1, 130, 512), (1, 1, 5, 3), (2, 1, 300, 20)])
@pytest.mark.parametrize("sharp", [1.0, 6.0], ids=["plain", "sharp"])
def test_attention_on_tensor_cores(heads, kv_heads, dim, vdim, sharp):
    """Portions of 32 and more tokens take the tcgen05 kernel (128-row tiles of (token, head) pairs: groups that divide 128 and that do
    not, one and two CTAs per SM, one and two groups of value columns, queries in tensor memory and in shared memory), single tokens
    and short portions the mma.sync kernel with key shares; along one sequence all of them must agree with the restatement.  With
    sharpened queries a lost or misplaced key would show far above the bound of bf16 operands."""
    layers = [layer(parallel(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=dim ** -0.5, temp=(0.3, 50)))]
    spec, w = make(layers, width=64, vocab=96, seed=43, tweak=lambda w: (sharpen(sharp)(w), only("right", w)))
    toks = tokens_of(spec, 400, 44)
    ref = oracle_logits(spec, w, toks)
    eng = engine(spec, w, exact_f32=False)
    try:
        got = feed_cut(eng, "a", toks, [190, 1, 1, 62, 1, 32, 33, 1, 5, 1, 70, 1])
        assert rel(got, ref) < TOL16
        whole = eng.feed([("w", toks, list(range(len(toks))))])
        assert rel(whole, ref) < TOL16
        if sharp > 1:                                          # the test has teeth: another key at one place is outside the bound
            other = list(toks)
            other[63] = (other[63] + 1) % spec.vocab
            assert rel(oracle_logits(spec, w, other)[64:], ref[64:]) > 1.5 * TOL16
    finally:
        eng.close()


@pytest.mark.parametrize("heads,dim,vdim,rot", [(3, 16, 16, 8), (2, 128, 128, 128), (2, 64, 128, 0), (4, 96, 64, 48), (3, 33, 20, 10), (2, 40, 200, 40),
                                                (1, 128, 256, 64), (1, 1, 1, 0), (2, 160, 64, 32)])
def test_retention_in_runs(heads, dim, vdim, rot):
    """Portions of 32 and more tokens go through runs of up to 128 tokens on tcgen05 (sizes beyond it through the token-by-token rule),
    single tokens through the one-pass kernel: lengths around one and several runs, states carried from portion to portion, decays
    from forgetting at once to keeping everything."""
    layers = [layer(parallel(rheads=heads, rdim=dim, rvdim=vdim, rot=rot, base=5e3, decay=[0.25, 1.0, 0.97, 0.9995][:heads]))]
    spec, w = make(layers, width=64, vocab=96, seed=53, tweak=lambda w: only("left", w))
    toks = tokens_of(spec, 500, 54)
    ref = oracle_logits(spec, w, toks)
    eng = engine(spec, w, exact_f32=False)
    try:
        for cuts in ([500], [127, 1, 128, 1, 129, 1, 33, 1], [1, 32, 64, 1, 65, 31, 200, 1, 2]):
            assert rel(feed_cut(eng, "a", toks, cuts), ref) < TOL16, cuts
            eng.close_session("a")
    finally:
        eng.close()


def test_unequal_requests_on_tensor_cores():
    """Portions of several requests in one step (runs and query tiles that start anywhere in a page, partly filled ones, odd numbers
    of them, a later request's beside an earlier one's) beside single tokens of others."""
    layers = [layer(parallel(heads=6, kv_heads=2, dim=64, vdim=32, scale=0.2, rdim=64, rvdim=64, rot=32), moe(ff=64, experts=4, top=4)),
              layer(parallel(heads=4, kv_heads=4, dim=32, vdim=96, rdim=32, rvdim=160), dense(ff=128))]
    spec, w = make(layers, width=128, vocab=128, seed=47, loop=(0, 2, 2))
    eng = engine(spec, w, exact_f32=False, num_pages=24, max_batched_tokens=704, debug_logit_rows=704)
    try:
        seqs = {n: tokens_of(spec, ln, 80 + i) for i, (n, ln) in enumerate([("a", 330), ("b", 170), ("c", 90), ("d", 260)])}
        plan = [{"a": 100, "b": 40}, {"a": 1, "b": 65, "c": 37}, {"a": 130, "b": 1, "c": 1, "d": 129}, {"a": 33, "c": 50, "d": 1},
                {"a": 64, "b": 64, "c": 2, "d": 130}, {"a": 2}]
        got = run_plan(eng, seqs, plan)
        for n, t in seqs.items():
            ref = oracle_logits(spec, w, t)
            assert rel(got[n], ref) < TOL16, n
            eng.close_session(n)
            assert rel(eng.feed([(n + "-alone", t, list(range(len(t))))]), got[n]) < TOL16
            eng.close_session(n + "-alone")
    finally:
        eng.close()


@pytest.mark.parametrize("exact", [False, True], ids=["tensor-cores", "exact-fp32"])
def test_projections_and_experts_on_tensor_cores(exact):
    """Shapes that tile: from nine rows on the input, pass, output and feed-forward projections run on tcgen05 from bf16 hi + lo planes,
    and the experts from 256 (token, choice) pairs; biases and clipped products go through the planes kernel."""
    layers = [layer(parallel(heads=4, kv_heads=2, dim=32, vdim=32, rdim=32, rvdim=32, rheads=4, decay=[0.5, 0.9, 0.99, 1.0]), dense(ff=192)),
              layer(parallel(heads=2, kv_heads=1, dim=64, vdim=64, rdim=64, rvdim=64, rheads=2), moe(ff=64, experts=4, top=4, limit=0.8))]
    spec, w = make(layers, width=128, vocab=256, seed=37, loop=(0, 2, 2))
    eng = engine(spec, w, exact_f32=exact)
    try:
        toks = tokens_of(spec, 400, 38)
        got = feed_cut(eng, "a", toks, [300, 1, 1, 12, 3, 10, 1, 60, 1])
        assert rel(got, oracle_logits(spec, w, toks)) < (TOL if exact else TOL16)
    finally:
        eng.close()


@pytest.mark.parametrize("experts,top,ff,skew", [(4, 1, 64, False), (40, 3, 64, False), (70, 2, 128, False), (40, 2, 64, True)],
                         ids=["few", "forty", "seventy", "skewed"])
def test_many_experts_in_one_launch(experts, top, ff, skew):
    """Experts with no pair, a few pairs and several tiles of 128 pairs in one launch, tiles found from the segment table across more
    than one warp's worth of experts.  The mixer adds nothing here, so the router sees what the restatement sees and no choice is close."""
    def tweak(w):
        only("left", w)
        only("right", w)
    spec, w = make([layer(parallel(), moe(ff=ff, experts=experts, top=top, limit=0.9))], width=128, vocab=256, seed=61, tweak=tweak)
    toks = [11] * 430 + tokens_of(spec, 70, 62) if skew else tokens_of(spec, 500, 62)
    ref = oracle_logits(spec, w, toks)
    eng = engine(spec, w, exact_f32=False)
    try:
        assert rel(eng.feed([("a", toks, list(range(500)))]), ref) < 4e-4
        assert rel(feed_cut(eng, "b", toks, [300, 1, 9, 130, 2, 58]), ref) < 4e-4
    finally:
        eng.close()


# ------------------------------------------------------------------------------------------------ the serving path
def greedy_oracle(spec, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(oracle_logits(spec, w, toks)[-1].argmax()))
    return toks[len(prompt):]


def test_greedy_generation_through_the_scheduler():
    """Engine.generate: submit -> the scheduler's own chunked prefill and decode steps -> argmax sampling; three requests
    of unequal length run together, prompts longer than a step's token budget are cut by the scheduler itself."""
    spec, w = make(MIXED, seed=23, loop=LOOP)
    eng = engine(spec, w, max_batched_tokens=48, decode_prefill_cap=16)
    try:
        prompts = [tokens_of(spec, ln, 60 + i) for i, ln in enumerate([100, 7, 51])]
        got = eng.generate(prompts, 12, temperature=0.0, ignore_eos=True)
        for p, g in zip(prompts, got):
            assert g == greedy_oracle(spec, w, p, 12)
        # a conversation that continues keeps its pages and states; one that diverges starts over
        eng.close()
        eng = engine(spec, w, max_batched_tokens=48, decode_prefill_cap=16)
        first = eng.generate([prompts[1]], 5, sessions=["gen-1"], temperature=0.0, ignore_eos=True)[0]
        more = prompts[1] + first + tokens_of(spec, 6, 99)
        assert eng.generate([more], 4, sessions=["gen-1"], temperature=0.0, ignore_eos=True)[0] == greedy_oracle(spec, w, more, 4)
        assert eng.stats()["prefix_hit_tokens"] > 0
        other = prompts[1][:4] + tokens_of(spec, 9, 98)
        assert eng.generate([other], 3, sessions=["gen-1"], temperature=0.0, ignore_eos=True)[0] == greedy_oracle(spec, w, other, 3)
    finally:
        eng.close()


def test_sampling_with_temperature_runs():
    spec, w = make(MIXED, seed=25, loop=LOOP)
    eng = engine(spec, w, exact_f32=False)
    try:
        out = eng.generate([tokens_of(spec, 20, 1), tokens_of(spec, 5, 2)], 8, temperature=0.8, top_k=20, top_p=0.9, ignore_eos=True)
        assert [len(o) for o in out] == [8, 8] and all(0 <= t < spec.vocab for o in out for t in o)
    finally:
        eng.close()


def test_trace_runner_replays_a_schedule(tmp_path):
    """bin/trace_run on a saved checkpoint: three steps, a session pausing and two ending, in both number formats."""
    from fasttalk_llm_microservice_b200.layered import save_checkpoint
    layers = [layer(parallel(), dense()), layer(parallel(kv_heads=4), moe(experts=3, top=3))]
    spec, w = make(layers, seed=31, loop=(0, 2, 2))
    save_checkpoint(spec, w, str(tmp_path / "model"))
    toks = tokens_of(spec, 60, 3)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:50], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[50:51], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[51:], "want": [8]}, {"id": "y", "tokens": toks[:5], "want": [4]}],
              "end": ["x", "y"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / ("out-" + dtype)
        r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "model"), "--dtype", dtype,
                            "--out", str(out), "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                           capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
        ref = oracle_logits(spec, w, toks)
        a = np.fromfile(out / "0.f32", dtype="<f4").reshape(2, spec.vocab)
        c = np.fromfile(out / "2.f32", dtype="<f4").reshape(2, spec.vocab)
        assert not (out / "1.f32").exists()
        tol = TOL if dtype == "float32" else TOL16
        assert rel(a, ref[[0, 29]]) < tol and rel(c[0], ref[59]) < tol and rel(c[1], ref[4]) < tol


def test_served_through_the_handler(tmp_path, monkeypatch):
    """A Fedutar checkpoint behind the serving path: FASTTALK_CHECKPOINT -> registry -> engine -> NativeHandler streams text."""
    from fasttalk_llm_microservice_b200.handler import NativeHandler, build_runner
    from fasttalk_llm_microservice_b200.layered import save_checkpoint
    spec, w = make([layer(parallel(), dense()), layer(parallel(), moe())], width=64, vocab=600, seed=41, loop=(0, 1, 2))
    save_checkpoint(spec, w, str(tmp_path / "ckpt"))
    monkeypatch.setenv("FASTTALK_CHECKPOINT", str(tmp_path / "ckpt"))
    monkeypatch.setenv("FASTTALK_ALLOW_BYTE_TOKENIZER", "1")
    monkeypatch.setenv("FASTTALK_MAX_SESSIONS", "4")
    monkeypatch.setenv("FASTTALK_MAX_CONTEXT", "512")
    monkeypatch.setenv("FASTTALK_MAX_BATCHED_TOKENS", "256")
    runner = build_runner("fedutar-test")
    h = NativeHandler(model="fedutar-test", runner=runner)
    try:
        assert h.check_connection()
        chunks = list(h.generate_stream([{"role": "user", "content": "hello there"}], temperature=0.0, max_tokens=12,
                                        request_id="conv-1"))
        assert 1 <= len(chunks) <= 12
        st = h.runner.engine.stats()
        assert st["prefill_tokens"] > 0 and st["decode_tokens"] > 0
    finally:
        h.close()
        runner.shutdown()
        runner.engine.close()
