"""CPU side of the Fedutar design: config <-> spec, layer runs, checkpoint files, the family registry, the packed descriptors, and
properties of the plain restatement (oracle/fedutar_oracle.py) that the GPU tests lean on."""
import json
import math

import pytest
import torch

from fasttalk_llm_microservice_b200 import layered as LY
from fasttalk_llm_microservice_b200.registry import family_of, load_model
from oracle import fedutar_oracle as O


def mixer(heads=4, kv_heads=2, dim=6, vdim=5, q_temp=True, rheads=3, rdim=8, rvdim=7, rot=6, ls=0.7, rs=1.1):
    left = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": 0.37, "vdim": vdim}
    if q_temp:
        left["q_temp"] = {"coef": 0.2, "every": 5}
    right = {"decay": [1.0 - 2.0 ** -(2 + h) for h in range(rheads)], "dim": rdim, "heads": rheads, "vdim": rvdim}
    if rot:
        right["rot"] = {"base": 700.0, "dims": rot}
    return {"left": left, "left_scale": ls, "right": right, "right_scale": rs}


def small_config():
    return {"architecture": "Fedutar", "embedding": {"scale": 3.0}, "logit_scale": 0.25, "logit_softcap": 12.0,
            "loop": {"start": 1, "stop": 3, "times": 2}, "norm": {"eps": 1e-5}, "vocab": 60, "width": 28, "layers": [
                {"type": "parallel", "mixer": mixer(), "mlp": {"ff": 10, "kind": "dense"}},
                {"type": "parallel", "mixer": mixer(heads=3, kv_heads=3, q_temp=False, rot=0),
                 "mlp": {"expert": {"ff": 12, "limit": 2.5}, "kind": "moe", "router": {"experts": 5, "top": 2}}},
                {"type": "parallel", "mixer": mixer(rot=8), "mlp": None},
                {"type": "parallel", "mixer": mixer(heads=2, kv_heads=1), "mlp": {"expert": {"ff": 6, "limit": 0.5}, "kind": "moe",
                                                                                  "router": {"experts": 3, "top": 3}}}]}


def small_spec():
    cfg = small_config()
    return cfg, LY.spec_from_config(cfg, None, name="t")


def test_config_roundtrip_shapes_and_runs():
    cfg, spec = small_spec()
    assert spec.config() == cfg and all(l.form == "sandwich" and l.plain_gain for l in spec.layers)
    shapes = LY.tensor_shapes(spec)
    assert LY.spec_from_config(cfg, shapes, name="t") == spec
    assert "head" not in shapes and shapes["loop.in"] == (28, 56) and shapes["final.norm"] == (28,)
    assert shapes["l0.mix.left.q"] == (24, 28) and shapes["l0.mix.left.k"] == (12, 28) and shapes["l0.mix.left.v"] == (10, 28)
    assert shapes["l0.mix.left.q.norm"] == (6,) == shapes["l0.mix.left.k.norm"] and shapes["l0.mix.left.g"] == (20, 28)
    assert shapes["l0.mix.right.q"] == (24, 28) == shapes["l0.mix.right.k"] and shapes["l0.mix.right.v"] == (21, 28)
    assert shapes["l0.mix.right.g"] == (21, 28) and shapes["l0.mix.right.o"] == (28, 21) and "l0.mix.right.norm" not in shapes
    assert shapes["l0.mlp.gate.b"] == (10,) and shapes["l0.mlp.down.b"] == (28,) and "l1.mlp.e0.gate.b" not in shapes
    assert shapes["l1.mlp.e4.gate"] == (12, 28) and shapes["l1.mlp.router"] == (5, 28) and "l2.norm2" not in shapes
    assert [i for i, _ in spec.runs()] == [0, 1, 2, 1, 2, 3] and [(i, t is not None) for i, t in spec.runs()] == O.runs(cfg)
    for loop in (None, {"start": 0, "stop": 4, "times": 1}, {"start": 0, "stop": 1, "times": 3}, {"start": 3, "stop": 4, "times": 2}):
        c = {**cfg, "loop": loop} if loop else {k: v for k, v in cfg.items() if k != "loop"}
        s = LY.spec_from_config(c)
        assert [(i, t is not None) for i, t in s.runs()] == O.runs(c) and s.config() == c and ("loop.in" in LY.tensor_shapes(s)) == bool(loop)
    bare = {k: v for k, v in cfg.items() if k not in ("logit_softcap", "loop")}
    assert LY.spec_from_config(bare).logit_softcap == 0.0 and LY.spec_from_config(bare).config() == bare
    for broken in (lambda c: c["layers"][0].update(type="mamba2"), lambda c: c["layers"][1].update(mlp={"kind": "sparse"}),
                   lambda c: c["loop"].update(stop=5), lambda c: c["layers"][0]["mixer"]["right"]["decay"].append(0.5),
                   lambda c: c["layers"][0]["mixer"]["right"]["rot"].update(dims=10)):
        bad = small_config()
        broken(bad)
        with pytest.raises(ValueError):
            LY.spec_from_config(bad)


def test_checkpoint_files_and_registry(tmp_path):
    _, spec = small_spec()
    w = LY.init_weights(spec, seed=1)
    LY.save_checkpoint(spec, w, str(tmp_path))
    with open(tmp_path / "config.json") as f:
        assert family_of(json.load(f)) == "layered"
    spec2, w2 = load_model(str(tmp_path), name="t")
    assert spec2 == spec and all(torch.equal(w[k], w2[k]) for k in w)
    bad = dict(w)
    del bad["l1.mlp.e2.gate"]
    LY.save_checkpoint(spec, bad, str(tmp_path / "bad"))
    with pytest.raises(KeyError):
        LY.load_checkpoint(str(tmp_path / "bad"))


def test_packed_descriptors():
    _, spec = small_spec()
    w = LY.init_weights(spec, seed=2)
    model, keep = LY.pack(spec, w, "cpu")
    by_ptr = {t.data_ptr(): t for t in keep if isinstance(t, torch.Tensor)}
    f32 = lambda n: w[n].float()
    assert model.n_layers == 6 and abs(model.embed_scale - 3.0) < 1e-6 and model.head == model.embed and model.logit_softcap == 12.0
    assert torch.allclose(by_ptr[model.final_norm_w], 0.25 * f32("final.norm"))            # the logits' factor is in the last gain
    d = [model.layers[i] for i in range(6)]
    assert all(x.form == LY.LAYER_SANDWICH and x.mixer == LY.MIXER_BRANCHES and x.n_branches == 2 for x in d)
    assert d[1].w_in == d[3].w_in and d[2].w_in == d[4].w_in                               # a layer that runs again shares its weights
    assert [bool(x.pass_in) for x in d] == [False, True, False, True, False, False] and torch.equal(by_ptr[d[1].pass_in], w["loop.in"])
    assert torch.equal(by_ptr[d[0].norm_pre1], f32("l0.norm1")) and torch.equal(by_ptr[d[0].norm_post2], f32("l0.norm2b"))
    a, r = d[0].branch[0], d[0].branch[1]
    w_in = by_ptr[d[0].w_in]
    assert d[0].n_in % 128 == 0 and all(o % 4 == 0 for o in (a.o_q, a.o_k, a.o_v, a.o_g, r.o_q, r.o_g))
    assert torch.equal(w_in[a.o_q:a.o_q + 24], w["l0.mix.left.q"]) and torch.equal(w_in[a.o_v:a.o_v + 10], w["l0.mix.left.v"])
    assert torch.equal(w_in[a.o_g:a.o_g + 20], w["l0.mix.left.g"]) and torch.equal(w_in[r.o_k:r.o_k + 24], w["l0.mix.right.k"])
    assert torch.equal(w_in[r.o_v:r.o_v + 21], w["l0.mix.right.v"]) and torch.equal(w_in[r.o_g:r.o_g + 21], w["l0.mix.right.g"])
    assert (a.kind, a.heads, a.kv_heads, a.window, a.rot_dims, a.qk_norm, a.tensor_cache) == (LY.BRANCH_WINDOW_ATTENTION, 4, 2, 0, 0, 1, 1)
    assert abs(a.q_temp_coef - 0.2) < 1e-7 and a.q_temp_every == 5 and abs(a.scale - 0.37) < 1e-7 and abs(a.out_scale - 0.7) < 1e-7
    assert torch.equal(by_ptr[a.q_gain], f32("l0.mix.left.q.norm")) and d[1].branch[0].q_temp_every == 0
    assert (r.kind, r.plain_qkv, r.head_norm, r.gate_act, r.rot_half, r.rot_dims) == (LY.BRANCH_DECAY_ATTENTION, 1, 1, 1, 1, 6)
    assert abs(r.k_scale - 8 ** -0.5) < 1e-7 and not r.out_norm and d[1].branch[1].rot_dims == 0 and not d[1].branch[1].rot_freq
    assert torch.allclose(by_ptr[r.rot_freq], torch.tensor([700.0 ** (-2 * i / 6) for i in range(3)]))
    assert torch.allclose(by_ptr[r.decay], torch.tensor([0.75, 0.875, 0.9375]))
    assert (d[0].ff_kind, d[0].ff_act, d[0].ff) == (LY.FF_DENSE, LY.ACT_SWIGLU, 10)
    assert torch.equal(by_ptr[d[0].gu_bias][1::2], f32("l0.mlp.up.b")) and torch.equal(by_ptr[d[0].down_bias], f32("l0.mlp.down.b"))
    e = d[1]
    assert (e.ff_kind, e.ff_act, e.experts, e.top, e.route_kind, e.route_norm) == (LY.FF_MOE, LY.ACT_CLIPPED_GLU, 5, 2, LY.ROUTE_SOFTMAX, 1)
    assert e.act_limit == 2.5 and abs(e.act_alpha - 1.702) < 1e-6 and e.act_shift == 1.0 and not e.gu_bias
    assert torch.equal(by_ptr[e.w_gu][3][0::2], w["l1.mlp.e3.gate"]) and d[2].ff_kind == LY.FF_NONE and d[5].act_limit == 0.5


def test_oracle_attention_temperature_and_groups():
    torch.manual_seed(0)
    f64 = torch.float64
    t = O.temperature(12, 0.3, 4, f64)
    assert torch.allclose(t[:3], torch.ones(3, dtype=f64)) and abs(t[3] - (1 + 0.3 * math.log(2))) < 1e-12      # p + 1 = 4 is the first step
    assert t[6] == t[3] and abs(t[7] - (1 + 0.3 * math.log(3))) < 1e-12 and abs(t[11] - (1 + 0.3 * math.log(4))) < 1e-12
    q, k, v = torch.randn(5, 4, 6, dtype=f64), torch.randn(5, 2, 6, dtype=f64), torch.randn(5, 2, 3, dtype=f64)
    o = O.causal_attention(q, k, v, 0.5).reshape(5, 4, 3)
    assert torch.allclose(o[0, 1], v[0, 0]) and torch.allclose(o[0, 2], v[0, 1])          # heads 0, 1 read key head 0; 2, 3 key head 1
    p = torch.softmax(0.5 * (k[:4, 1] @ q[3, 3]), 0)
    assert torch.allclose(o[3, 3], p @ v[:4, 1])


def test_oracle_retention_rotation_and_experts():
    torch.manual_seed(1)
    f64 = torch.float64
    x = torch.randn(5, 2, 8, dtype=f64)
    r = O.turn_halves(x, torch.arange(5), 6, 100.0)
    assert torch.equal(r[..., 6:], x[..., 6:]) and torch.allclose(r[0], x[0])
    s = torch.tensor(3.0 * 100.0 ** (-2.0 / 6.0), dtype=f64)                               # pair (1, 4) at position 3
    assert torch.allclose(r[3, 0, 1], x[3, 0, 1] * torch.cos(s) - x[3, 0, 4] * torch.sin(s))
    assert torch.allclose(r[3, 0, 4], x[3, 0, 4] * torch.cos(s) + x[3, 0, 1] * torch.sin(s))
    q, k, v = (torch.randn(6, 2, n, dtype=f64) for n in (8, 8, 3))
    o = O.retain(q, k, v, [0.5, 0.9])
    for h, d in ((0, 0.5), (1, 0.9)):                                                       # the sum written out
        want = sum(d ** (4 - j) * (q[4, h] @ k[j, h]) * v[j, h] for j in range(5))
        assert torch.allclose(o[4, h], want)
    w = {"gate": torch.randn(4, 3, dtype=f64), "up": torch.randn(4, 3, dtype=f64), "down": torch.eye(4, dtype=f64)}
    h = 10.0 * torch.randn(50, 3, dtype=f64)
    y = O.clipped_expert(h, w, "", 2.0)
    g, u = h @ w["gate"].T, h @ w["up"].T
    both = (g > 2.0) & (u > 2.0)
    top = 2.0 / (1.0 + math.exp(-1.702 * 2.0)) * 3.0
    assert both.any() and torch.allclose(y[both], torch.full_like(y[both], top))
    low = (g < -9.0) & (u < -2.0)                                                           # the gate has no lower limit, u + 1 = -1
    assert low.any() and torch.allclose(y[low], -(g * torch.sigmoid(1.702 * g))[low])


def test_oracle_is_causal_and_passes_start_from_the_join():
    cfg, spec = small_spec()
    w = LY.init_weights(spec, seed=3)
    toks = torch.randint(0, spec.vocab, (30,)).tolist()
    with torch.no_grad():
        full = O.forward(cfg, w, toks)
        assert torch.allclose(full[:17], O.forward(cfg, w, toks[:17]), atol=1e-9) and full.abs().max() <= 12.0
        changed = O.forward(cfg, w, [(toks[0] + 1) % spec.vocab] + toks[1:])
        assert (full[-1] - changed[-1]).abs().max() > 1e-6
        trail = []
        O.forward(cfg, w, toks, trail=trail)
        assert len(trail) == 6
        wd = {k: v.double() for k, v in w.items()}
        first = wd["embed"][torch.tensor(toks)] * 3.0
        a, b = wd["loop.in"][:, :28], wd["loop.in"][:, 28:]
        again = O.layer(trail[2] @ a.T + first @ b.T, wd, 1, cfg["layers"][1], 1e-5)
        assert torch.allclose(again, trail[3])
        assert torch.allclose(O.layer(trail[0] @ a.T + first @ b.T, wd, 1, cfg["layers"][1], 1e-5), trail[1])
