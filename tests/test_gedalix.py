"""CPU side of the Gedalix design: config <-> spec, layer runs, checkpoint files, the family registry, the packed descriptors, and
properties of the plain restatement (oracle/gedalix_oracle.py) that the GPU tests lean on."""
import json

import pytest
import torch

from fasttalk_llm_microservice_b200 import layered as LY
from fasttalk_llm_microservice_b200.registry import family_of, load_model
from oracle import gedalix_oracle as O


def small_config():
    a = {"dim": 6, "heads": 3, "kv_rank": 11, "rot": {"base": 500.0, "dims": 4}, "rot_dim": 4, "scale": 0.3, "vdim": 5}
    b = {"dim": 8, "heads": 2, "kv_rank": 32, "rot_dim": 0, "scale": 0.25, "vdim": 7}
    return {"architecture": "Gedalix", "embedding": {"scale": 3.0}, "loop": {"start": 1, "stop": 3, "times": 2}, "max_positions": 50,
            "norm": {"eps": 1e-5}, "residual_mult": 0.4, "vocab": 60, "width": 28, "layers": [
        {"type": "latent_attention", "mixer": dict(a), "mlp": None},
        {"type": "latent_attention", "mixer": dict(b),
         "mlp": {"expert": {"ff": 12}, "kind": "moe", "router": {"experts": 5, "top": 2}, "shared": {"ff": 9}}},
        {"type": "latent_attention", "mixer": dict(a), "mlp": {"expert": {"ff": 6}, "kind": "moe", "router": {"experts": 3, "top": 3}}},
        {"type": "latent_attention", "mixer": dict(b), "mlp": None}]}


def small_spec():
    cfg = small_config()
    return cfg, LY.spec_from_config(cfg, None, name="t")


def test_config_roundtrip_shapes_and_runs():
    cfg, spec = small_spec()
    assert spec.config() == cfg and [l.form for l in spec.layers] == ["prenorm"] * 4
    shapes = LY.tensor_shapes(spec)
    assert LY.spec_from_config(cfg, shapes, name="t") == spec
    assert shapes["pos"] == (50, 28) and shapes["loop.step"] == (2, 28) and shapes["head"] == (60, 28) and shapes["final.norm"] == (28,)
    assert shapes["l0.mix.q"] == (30, 28) and shapes["l0.mix.dkv"] == (15, 28) and shapes["l0.mix.uk"] == (18, 11)
    assert shapes["l0.mix.uv"] == (15, 11) and shapes["l0.mix.g"] == (15, 28) and shapes["l0.mix.sink"] == (3,) and "l0.norm2" not in shapes
    assert shapes["l1.mix.q"] == (16, 28) and shapes["l1.mix.dkv"] == (32, 28) and shapes["l1.mlp.router.b"] == (5,)
    assert shapes["l1.mlp.shared.sg"] == (1, 28) and shapes["l1.mlp.shared.up"] == (9, 28) and "l2.mlp.shared.sg" not in shapes
    assert spec.runs() == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)] == O.runs(cfg)
    for loop in (None, {"start": 0, "stop": 4, "times": 1}, {"start": 0, "stop": 1, "times": 3}, {"start": 3, "stop": 4, "times": 2}):
        c = {**cfg, "loop": loop} if loop else {k: v for k, v in cfg.items() if k != "loop"}
        s = LY.spec_from_config(c)
        assert s.runs() == O.runs(c) and s.config() == c and ("loop.step" in LY.tensor_shapes(s)) == bool(loop)
    for broken in (lambda c: c["layers"][0].update(type="mamba2"), lambda c: c["layers"][1].update(mlp={"kind": "sparse"}),
                   lambda c: c["loop"].update(stop=5), lambda c: c["layers"][0]["mixer"].update(rot_dim=6)):
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
    del bad["l1.mlp.shared.sg"]
    LY.save_checkpoint(spec, bad, str(tmp_path / "bad"))
    with pytest.raises(KeyError):
        LY.load_checkpoint(str(tmp_path / "bad"))


def test_packed_descriptors():
    _, spec = small_spec()
    w = LY.init_weights(spec, seed=2)
    model, keep = LY.pack(spec, w, "cpu")
    by_ptr = {t.data_ptr(): t for t in keep if isinstance(t, torch.Tensor)}
    assert model.n_layers == 6 and model.max_positions == 50 and abs(model.embed_scale - 3.0) < 1e-6
    assert torch.equal(by_ptr[model.pos_embed], w["pos"]) and torch.equal(by_ptr[model.final_norm_w], w["final.norm"].float())
    d = [model.layers[i] for i in range(6)]
    assert all(x.form == LY.LAYER_PRENORM and x.mixer == LY.MIXER_LATENT_ATTENTION and x.gate_wide == 1 for x in d)
    # both passes share their weights; the second takes the embedding output again, each its own vector at its first layer
    assert d[1].w_in == d[3].w_in and d[2].w_down == d[4].w_down and [x.re_embed for x in d] == [0, 0, 0, 1, 0, 0]
    assert torch.equal(by_ptr[d[1].pre_add], w["loop.step"][0].float()) and torch.equal(by_ptr[d[3].pre_add], w["loop.step"][1].float())
    assert not d[0].pre_add and not d[2].pre_add and not d[4].pre_add and not d[5].pre_add
    a, b = d[0], d[1]
    assert (a.heads, a.dim, a.vdim, a.kv_rank, a.rot_dims, a.ff_kind) == (3, 6, 5, 11, 4, LY.FF_NONE) and not a.norm_pre2
    w_in = by_ptr[a.w_in]
    assert a.n_in % 128 == 0 and torch.equal(w_in[a.o_q:a.o_q + 30], w["l0.mix.q"]) and torch.equal(w_in[a.o_dkv:a.o_dkv + 15], w["l0.mix.dkv"])
    assert torch.equal(w_in[a.o_gate:a.o_gate + 15], w["l0.mix.g"]) and a.o_dkv % 4 == 0 and a.o_gate % 4 == 0
    assert torch.allclose(by_ptr[a.rot_freq], torch.tensor([1.0, 500.0 ** -0.5])) and not b.rot_freq
    assert torch.allclose(by_ptr[a.res_gain[0]], 0.4 * w["l0.ls1"].float()) and torch.equal(by_ptr[a.sink], w["l0.mix.sink"].float())
    assert torch.equal(by_ptr[a.w_uk_t][2], w["l0.mix.uk"][12:18].T)
    assert (b.ff_kind, b.experts, b.top, b.ff, b.shared_ff, b.shared_gate) == (LY.FF_MOE, 5, 2, 12, 9, 1)
    assert (b.route_kind, b.route_norm, b.ff_act) == (LY.ROUTE_SOFTMAX, 1, LY.ACT_SWIGLU)
    assert torch.equal(by_ptr[b.w_router][5], w["l1.mlp.shared.sg"][0]) and torch.equal(by_ptr[b.router_bias], w["l1.mlp.router.b"].float())
    assert torch.equal(by_ptr[b.w_gu][4][1::2], w["l1.mlp.e4.up"]) and torch.equal(by_ptr[b.w_shared_up][0::2], w["l1.mlp.shared.gate"])
    assert d[2].shared_gate == 0 and d[2].shared_ff == 0 and d[2].top == 3


def test_oracle_attention_rotation_sink_and_routing():
    torch.manual_seed(0)
    f64 = torch.float64
    x = torch.randn(5, 2, 6, dtype=f64)
    r = O.turn_halves(x, torch.arange(5), 100.0)
    assert torch.allclose(r[0], x[0]) and torch.allclose((r * r).sum(-1), (x * x).sum(-1))
    s = torch.tensor(3.0 * 100.0 ** (-2.0 / 6.0), dtype=f64)               # pair (1, 4) at position 3
    assert torch.allclose(r[3, 0, 1], x[3, 0, 1] * torch.cos(s) - x[3, 0, 4] * torch.sin(s))
    assert torch.allclose(r[3, 0, 4], x[3, 0, 4] * torch.cos(s) + x[3, 0, 1] * torch.sin(s))
    q, k, v = (torch.randn(4, 2, n, dtype=f64) for n in (6, 6, 3))
    o = O.attend_with_sink(q, k, v, 0.5, torch.tensor([0.7, -1e9], dtype=f64)).reshape(4, 2, 3)
    e = torch.exp(0.5 * (q[0, 0] @ k[0, 0]))
    assert torch.allclose(o[0, 0], v[0, 0] * e / (e + torch.exp(torch.tensor(0.7, dtype=f64)))) and torch.allclose(o[0, 1], v[0, 1])
    w = {"router": torch.randn(6, 8, dtype=f64), "router.b": torch.zeros(6, dtype=f64)}
    h = torch.randn(9, 8, dtype=f64)
    ids, wt = O.choose(h, w, "", 2)
    z = h @ w["router"].T
    full = torch.softmax(z, -1)                              # softmax over the chosen logits = over all, divided by the chosen ones' sum
    assert torch.allclose(wt, full.gather(1, ids) / full.gather(1, ids).sum(-1, keepdim=True))
    w["router.b"][4] = 100.0
    assert (O.choose(h, w, "", 1)[0] == 4).all()


def test_oracle_is_causal_and_passes_differ():
    cfg, spec = small_spec()
    w = LY.init_weights(spec, seed=3)
    toks = torch.randint(0, spec.vocab, (30,)).tolist()
    with torch.no_grad():
        full = O.forward(cfg, w, toks)
        assert torch.allclose(full[:17], O.forward(cfg, w, toks[:17]), atol=1e-9)
        changed = O.forward(cfg, w, [(toks[0] + 1) % spec.vocab] + toks[1:])
        assert (full[-1] - changed[-1]).abs().max() > 1e-6
        trail = []
        O.forward(cfg, w, toks, trail=trail)
        assert len(trail) == 6
        # a pass starts from the stream, the embedding output and its own vector
        first = O.embedding(toks, {k: v.double() for k, v in w.items()}, 3.0)
        wd = {k: v.double() for k, v in w.items()}
        again = O.layer(trail[2] + first + wd["loop.step"][1], wd, 1, cfg["layers"][1], 1e-5, 0.4)
        assert torch.allclose(again, trail[3])
