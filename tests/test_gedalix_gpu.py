"""The Gedalix design on the GPU against the plain restatement in oracle/gedalix_oracle.py.

Every test builds its own small configuration and random weights (none of them a published model's sizes).  Logits are
compared at EVERY position.  The exact engine computes in fp32 on the bf16 weights, so its bound is rounding: 1e-4 of the
largest logit.  The serving form keeps latents of whole 32-column pieces, queries and softmax weights in bf16, which bounds the
agreement there.
"""
import copy
import json
import os
import subprocess

import numpy as np
import pytest
import torch

from oracle import gedalix_oracle as O

pytestmark = pytest.mark.gpu
TOL = 1e-4
TOL16 = 2e-2


# ------------------------------------------------------------------------------------------------ configurations
def latent(heads=3, dim=20, vdim=12, kv_rank=40, rot=8, scale=0.25, base=900.0):
    m = {"dim": dim, "heads": heads, "kv_rank": kv_rank, "rot_dim": rot, "scale": scale, "vdim": vdim}
    if rot:
        m["rot"] = {"base": base, "dims": rot}
    return {"type": "latent_attention", "mixer": m}


def moe(ff=24, experts=6, top=2, shared=36):
    m = {"expert": {"ff": ff}, "kind": "moe", "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def layer(mixer, mlp=None):
    return {**copy.deepcopy(mixer), "mlp": mlp}


def make(layers, width=80, vocab=150, eps=1e-5, seed=0, embed_scale=3.0, mult=0.6, loop=None, positions=640, tweak=None):
    from fasttalk_llm_microservice_b200.layered import init_weights, spec_from_config, tensor_shapes
    cfg = {"architecture": "Gedalix", "embedding": {"scale": embed_scale}, "layers": copy.deepcopy(layers), "max_positions": positions,
           "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab, "width": width}
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


def sharpen(f):
    """Weights whose scores spread `f` times wider: the softmax rests on a few keys, a lost or misplaced one shows."""
    def tweak(w):
        for k in list(w):
            if k.endswith("mix.q"):
                w[k] = (w[k].float() * f).to(torch.bfloat16)
    return tweak


MIXED = [layer(latent(), moe()), layer(latent(heads=5, dim=12, vdim=16, kv_rank=28, rot=6, base=50.0), moe(ff=17, experts=4, top=3, shared=9)),
         layer(latent(heads=2, dim=8, vdim=30, kv_rank=64, rot=0)), layer(latent(heads=4, kv_rank=33, rot=2), moe(top=1, shared=0))]
LOOP = (1, 3, 2)


# ------------------------------------------------------------------------------------------------ every mechanism alone
@pytest.mark.parametrize("layers,loop", [
    ([layer(latent())], None),
    ([layer(latent(rot=0))], None),
    ([layer(latent(heads=1, dim=1, vdim=3, kv_rank=5, rot=2))], None),
    ([layer(latent(heads=7, dim=33, vdim=9, kv_rank=100, rot=30, base=1e6, scale=0.1))], None),
    ([layer(latent(heads=2, dim=8, vdim=8, kv_rank=300, rot=48))], None),
    ([layer(latent(), moe(shared=0))], None),
    ([layer(latent(), moe())], None),
    ([layer(latent(), moe(ff=7, experts=3, top=3, shared=50))], None),
    ([layer(latent(), moe(ff=20, experts=40, top=1, shared=4))], None),
    ([layer(latent()), layer(latent())], (0, 1, 1)),
    ([layer(latent()), layer(latent(), moe())], (0, 2, 3)),
    ([layer(latent()), layer(latent(), moe()), layer(latent(heads=2))], (1, 2, 4)),
    ([layer(latent(), moe()), layer(latent())], (1, 2, 2)),
    (MIXED, None),
    (MIXED, LOOP),
], ids=["latent", "unrotated", "tiny", "odd", "wide-latent", "experts", "experts-shared", "experts-all", "experts-many", "one-pass",
        "loop-all", "loop-middle", "loop-end", "mixed", "mixed-loop"])
def test_whole_prompt_matches_oracle(layers, loop):
    spec, w = make(layers, seed=3, loop=loop)
    eng = engine(spec, w)
    try:
        toks = tokens_of(spec, 150, 1)
        got = eng.feed([("s", toks, list(range(len(toks))))])
        assert rel(got, oracle_logits(spec, w, toks)) < TOL
    finally:
        eng.close()


@pytest.mark.parametrize("width,vocab,scale,mult,eps", [(70, 333, 1.0, 1.0, 1e-6), (33, 50, 9.0, 0.1, 1e-3), (132, 128, 0.5, 2.0, 1e-5)])
def test_other_sizes_and_constants(width, vocab, scale, mult, eps):
    spec, w = make(MIXED, width=width, vocab=vocab, embed_scale=scale, mult=mult, eps=eps, loop=(0, 2, 3), seed=9)
    eng = engine(spec, w)
    try:
        toks = tokens_of(spec, 90, 2)
        ref = oracle_logits(spec, w, toks)
        assert rel(eng.feed([("s", toks, list(range(len(toks))))]), ref) < TOL
        assert rel(feed_cut(eng, "c", toks, [1, 2, 1, 7, 1]), ref) < TOL
    finally:
        eng.close()


def test_residual_after_every_layer_run():
    """The stream after every run of every layer, before what comes ahead of the next pass."""
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
    """Leaving out one part changes the logits by far more than the bound, so the agreement with the restatement says that each
    of them is computed: the sink, rotation, output gate, router bias, shared expert and its gate, layer scale, residual
    multiplier, positions, step vectors, the embedding added again, the number of passes."""
    spec, w = make(MIXED, seed=5, loop=LOOP)
    eng = engine(spec, w)
    try:
        toks = tokens_of(spec, 160, 6)
        ref = oracle_logits(spec, w, toks)
        assert rel(feed_cut(eng, "a", toks, [100, 1, 1, 1, 50, 1]), ref) < TOL
    finally:
        eng.close()
    changes = {"l0.mix.sink": -60.0, "l2.mix.sink": -60.0, "l0.mlp.router.b": 0.0, "l1.mlp.shared.sg": 0.0, "l0.ls1": 1.0, "l1.ls2": 1.0,
               "l0.mix.g": 0.0, "l0.mlp.shared.down": 0.0, "pos": 0.0, "loop.step": 0.0}
    for name, value in changes.items():
        w2 = dict(w)
        w2[name] = torch.full_like(w[name], value)
        assert rel(oracle_logits(spec, w2, toks), ref) > 30 * TOL, name
    w2 = dict(w)
    w2["loop.step"] = w["loop.step"].clone()
    w2["loop.step"][0] = 0                              # the first pass has its vector too
    assert rel(oracle_logits(spec, w2, toks), ref) > 30 * TOL
    for path, value in ((("residual_mult",), 0.55), (("embedding", "scale"), 2.9), (("loop", "times"), 1), (("loop", "start"), 2),
                        (("layers", 0, "mixer", "rot", "base"), 700.0), (("layers", 1, "mixer", "scale"), 0.3)):
        cfg = spec.config()
        d = cfg
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        assert rel(oracle_logits(spec, w, toks, cfg), ref) > 30 * TOL, path


@pytest.mark.parametrize("exact", [True, False], ids=["exact-fp32", "tensor-cores"])
@pytest.mark.parametrize("sink", [-30.0, 2.0, 9.0, 200.0])
def test_sinks_below_among_and_far_above_the_scores(sink, exact):
    """A sink far below every score counts nothing; one among them takes its share (most of it at the first tokens, which see few
    keys); one far above them takes everything and leaves zeros, not infinities.  Different sinks per head."""
    def tweak(w):
        w["l0.mix.sink"][:] = torch.tensor([sink, sink / 2, -sink])
        w["l0.ls1"][:] = 3.0
    spec, w = make([layer(latent(heads=3, dim=16, vdim=32, kv_rank=64, rot=8))], width=64, seed=15, tweak=tweak)
    eng = engine(spec, w, exact_f32=exact)
    try:
        toks = tokens_of(spec, 150, 16)
        ref = oracle_logits(spec, w, toks)
        got = feed_cut(eng, "a", toks, [1, 1, 70, 1, 1, 60, 1])
        assert np.isfinite(got).all() and rel(got, ref) < (TOL if exact else TOL16)
        assert rel(eng.feed([("b", toks, list(range(150)))]), ref) < (TOL if exact else TOL16)
    finally:
        eng.close()


# ------------------------------------------------------------------------------------------------ portions, decoding
@pytest.mark.parametrize("cuts", [[1], [2], [3, 2, 29, 1, 1, 17, 2], [64], [63, 1, 1, 64, 2], [65, 2]],
                         ids=["token-by-token", "twos", "ragged", "pages", "around-pages", "over-a-page"])
def test_portions_and_decoding_match_the_whole_prompt(cuts):
    spec, w = make(MIXED, seed=7, loop=LOOP)
    eng = engine(spec, w)
    try:
        toks = tokens_of(spec, 200, 8)
        ref = oracle_logits(spec, w, toks)
        whole = eng.feed([("w", toks, list(range(len(toks))))])
        got = feed_cut(eng, "c", toks, cuts)
        assert rel(whole, ref) < TOL and rel(got, ref) < TOL
        assert rel(got, whole) < 2e-5
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


def marked(rot, width=64, rank=64):
    """Token 0 lives on coordinate 0 of the stream and token 1 on coordinate 1; the latent keeps them apart.  Every query points
    along channel 0; only token 1's key meets it (through the plain part, or with rot through the shared rotated part, whose
    slow pair hardly turns over the sequence)."""
    def tweak(w):
        for n in ("embed", "pos", "l0.mix.q", "l0.mix.dkv", "l0.mix.uk"):
            w[n][:] = 0
        w["embed"][0, 0] = w["embed"][1, 1] = 1.0
        w["l0.norm1"][:] = 1.0
        w["l0.mix.dkv.norm"][:] = 1.0
        w["l0.mix.dkv"][0, 0] = w["l0.mix.dkv"][1, 1] = 1.0
        w["l0.mix.sink"][:] = -2.0
        for h in range(3):
            qrow = h * (16 + rot)
            if rot:
                i = rot // 2 - 1                                      # the slowest pair: the first coordinate of it
                w["l0.mix.q"][qrow + 16 + i, 0] = w["l0.mix.q"][qrow + 16 + i, 1] = 1.0
                w["l0.mix.dkv"][rank + i, 1] = 1.0
            else:
                w["l0.mix.q"][qrow, 0] = w["l0.mix.q"][qrow, 1] = 1.0
                w["l0.mix.uk"][h * 16, 1] = 1.0
    return make([layer(latent(heads=3, dim=16, vdim=32, kv_rank=rank, rot=rot, base=1e6, scale=0.25))], width=width, vocab=40, seed=2,
                embed_scale=1.0, mult=1.0, positions=800, tweak=tweak)


@pytest.mark.parametrize("exact", [True, False], ids=["exact-fp32", "tensor-cores"])
@pytest.mark.parametrize("rot", [0, 16])
def test_one_far_key_among_hundreds(rot, exact):
    """One marked token in a sequence of equal tokens takes most of the weight for everyone after it, however far, and none
    before it; at and around page borders, in a prompt, in portions and in decoding."""
    spec, w = marked(rot)
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


@pytest.mark.parametrize("exact", [True, False], ids=["exact-fp32", "tensor-cores"])
def test_pages_are_used_again(exact):
    """A pool of 6 pages serves six sequences, one after the other and two at a time: what an ended session left in its pages
    (of every layer run) must not reach the next one."""
    # every expert chosen: bf16 attention must not meet a close choice
    layers = [layer(latent(heads=2, dim=16, vdim=16, kv_rank=32, rot=8, scale=1.0), moe(experts=3, top=3)),
              layer(latent(heads=3, kv_rank=64, rot=4, scale=1.0))]
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
            got = run_plan(eng, {f"s{a}": seqs[a], f"s{b}": seqs[b]}, [{f"s{a}": 37, f"s{b}": 20 if k == 0 else 1 + 34 * (k % 2)} for k in range(14)])
            for i in (a, b):
                assert rel(got[f"s{i}"], ref[i]) < tol
                eng.close_session(f"s{i}")
        st = eng.stats()
        assert st["free_pages"] == 6 and st["live_sessions"] == 0
    finally:
        eng.close()


def test_no_sequence_grows_beyond_the_position_table():
    from fasttalk_llm_microservice_b200.native import NativeError
    spec, w = make([layer(latent())], positions=70)
    eng = engine(spec, w)
    try:
        toks = tokens_of(spec, 71, 1)
        assert rel(feed_cut(eng, "a", toks[:70], [69, 1]), oracle_logits(spec, w, toks[:70])) < TOL
        with pytest.raises(NativeError):
            eng.feed([("a", toks[70:], [0])])
        assert len(eng.generate([toks[:66]], 20, temperature=0.0, ignore_eos=True)[0]) <= 5      # ends at the table's end
    finally:
        eng.close()


# ------------------------------------------------------------------------------------------------ tensor cores
@pytest.mark.parametrize("heads,rank,rot,dim,vdim", [(3, 32, 0, 32, 32), (16, 64, 16, 32, 64), (20, 96, 16, 16, 8), (1, 128, 64, 64, 32), (6, 160, 32, 32, 96),
                                                     (2, 256, 64, 128, 128), (5, 288, 30, 32, 32), (2, 512, 64, 64, 64), (40, 64, 8, 8, 8)])
@pytest.mark.parametrize("sharp", [1.0, 8.0], ids=["plain", "sharp"])
def test_latent_attention_on_tensor_cores(heads, rank, rot, dim, vdim, sharp):
    """Latents of whole 32-column pieces: portions of 32 and more tokens take the tcgen05 kernel (128-row tiles of (token, head)
    pairs: heads that divide 128 and that do not, one and two groups of value columns, queries in tensor memory and in shared
    memory), single tokens and short portions the mma.sync kernel with key shares; along one sequence all of them must agree with
    the restatement.  With sharpened queries a lost or misplaced key would show far above the bound of bf16 operands."""
    layers = [layer(latent(heads=heads, dim=dim, vdim=vdim, kv_rank=rank, rot=rot, scale=(dim + rot) ** -0.5, base=1e4))]
    spec, w = make(layers, width=64, vocab=96, seed=43, tweak=sharpen(sharp))
    toks = tokens_of(spec, 400, 44)
    ref = oracle_logits(spec, w, toks)
    eng = engine(spec, w, exact_f32=False)
    try:
        got = feed_cut(eng, "a", toks, [190, 1, 1, 62, 1, 32, 33, 1, 5, 1, 70, 1])
        assert rel(got, ref) < TOL16
        whole = eng.feed([("w", toks, list(range(len(toks))))])
        assert rel(whole, ref) < TOL16
        if sharp > 1:                                          # the test has teeth: one key more or less is far outside the bound
            cut = oracle_logits(spec, w, toks[1:])
            assert rel(cut[100:], ref[101:]) > 2 * TOL16
    finally:
        eng.close()


def test_unequal_requests_on_tensor_cores():
    """Portions of several requests in one step (query tiles of 64 tokens that start anywhere in a page, partly filled ones, a
    later one of the same step that sees another request's pages nowhere) beside single tokens of others."""
    layers = [layer(latent(heads=5, dim=64, vdim=32, kv_rank=64, rot=24, scale=0.5), moe(ff=64, experts=4, top=4, shared=64)),
              layer(latent(heads=3, dim=32, vdim=64, kv_rank=96, rot=8))]
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
    """Shapes that tile: from nine rows on the input, per-head, output and feed-forward projections run on tcgen05 from bf16 hi + lo
    planes, and the experts from 256 (token, choice) pairs.  A latent that is no multiple of 32 keeps the attention in fp32, so the
    two forms must agree closely along one sequence."""
    layers = [layer(latent(heads=4, dim=32, vdim=32, kv_rank=80, rot=16), moe(ff=64, experts=4, top=2, shared=128)),
              layer(latent(heads=2, dim=64, vdim=64, kv_rank=48, rot=8), moe(ff=128, experts=2, top=1, shared=64))]
    spec, w = make(layers, width=128, vocab=256, seed=37, loop=(1, 2, 2))
    eng = engine(spec, w, exact_f32=exact)
    try:
        toks = tokens_of(spec, 400, 38)
        got = feed_cut(eng, "a", toks, [300, 1, 1, 12, 3, 10, 1, 60, 1])
        assert rel(got, oracle_logits(spec, w, toks)) < (TOL if exact else 4e-4)
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
        # a conversation that continues keeps its pages; one that diverges drops what no longer matches
        eng.close()
        eng = engine(spec, w, max_batched_tokens=48, decode_prefill_cap=16)
        first = eng.generate([prompts[1]], 5, sessions=["gen-1"], temperature=0.0, ignore_eos=True)[0]
        more = prompts[1] + first + tokens_of(spec, 6, 99)
        assert eng.generate([more], 4, sessions=["gen-1"], temperature=0.0, ignore_eos=True)[0] == greedy_oracle(spec, w, more, 4)
        assert eng.stats()["prefix_hit_tokens"] > 0
        other = tokens_of(spec, 11, 98)
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
    spec, w = make(MIXED, seed=31, loop=LOOP)
    save_checkpoint(spec, w, str(tmp_path / "model"))
    toks = tokens_of(spec, 40, 3)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[30:31], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[31:], "want": [8]}, {"id": "y", "tokens": toks[:5], "want": [4]}],
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
        assert rel(a, ref[[0, 29]]) < tol and rel(c[0], ref[39]) < tol and rel(c[1], ref[4]) < tol


def test_served_through_the_handler(tmp_path, monkeypatch):
    """A Gedalix checkpoint behind the serving path: FASTTALK_CHECKPOINT -> registry -> engine -> NativeHandler streams text."""
    from fasttalk_llm_microservice_b200.handler import NativeHandler, build_runner
    from fasttalk_llm_microservice_b200.layered import save_checkpoint
    spec, w = make([layer(latent(), moe()), layer(latent(kv_rank=32))], width=64, vocab=600, seed=41, loop=(0, 1, 2))
    save_checkpoint(spec, w, str(tmp_path / "ckpt"))
    monkeypatch.setenv("FASTTALK_CHECKPOINT", str(tmp_path / "ckpt"))
    monkeypatch.setenv("FASTTALK_ALLOW_BYTE_TOKENIZER", "1")
    monkeypatch.setenv("FASTTALK_MAX_SESSIONS", "4")
    monkeypatch.setenv("FASTTALK_MAX_CONTEXT", "512")
    monkeypatch.setenv("FASTTALK_MAX_BATCHED_TOKENS", "256")
    runner = build_runner("gedalix-test")
    h = NativeHandler(model="gedalix-test", runner=runner)
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
