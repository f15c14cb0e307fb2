"""Pidodra without a GPU: configuration, the model description built from it
(cache needs, tensor names, which layers read another's cache), the random-weights
writer and the loader's one error; frequencies and the order of rotated rows; the
plain implementation against closed forms; and that the test models' weights make
every mechanism show."""

import copy
import math
import os

import numpy as np
import pytest

import pidodra_models as pm
import plain_pidodra as pp


def spec_of(cfg):
    from reflex_b200 import models  # noqa: F401
    from reflex_b200.config.registry import spec_from_config_dict

    return spec_from_config_dict(cfg)


def test_config_to_model_description():
    from reflex_b200.engine.model import expected_tensors

    typed, spec = spec_of(pm.PID_A)
    assert spec.architecture == "pidodra" and (spec.vocab_size, spec.hidden_size) == (97, 72)
    assert not spec.tie_word_embeddings and spec.embedding_norm is None and spec.embedding_scale == 2.5
    assert [l.block for l in spec.layers] == ["sum_norm"] * 5
    assert all(dict(l.params)["alpha"] == 1.5 for l in spec.layers)
    assert [l.mixer.kind for l in spec.layers] == ["latent_attention", "gqa_attention", "gqa_attention",
                                                   "latent_attention", "gqa_attention"]
    lat, a, b, _, c = (l.mixer for l in spec.layers)
    assert (lat.num_heads, lat.head_dim, lat.value_dim, lat.scale, lat.window) == (3, 16, 24, 0.6, None)
    assert [lat.param(k) for k in ("q_rank", "kv_rank", "rot_dim", "eps", "sink", "gate")] == [40, 24, 8, 1e-5, True, "element"]
    assert lat.position.kind == "rope_neox" and dict(lat.position.params)["pairing"] == "consecutive"
    assert (a.num_heads, a.num_kv_heads, a.head_dim, a.value_dim, a.scale) == (6, 3, 16, 24, 0.5)
    assert a.position.kind == "rope_yarn" and (a.position.rotary_dim, a.position.theta) == (8, 100.0)
    assert dict(a.position.params) == {"factor": 4.0, "original": 64.0, "fast": 8.0, "slow": 1.0}
    assert a.qk_norm.size == 16 and a.qk_norm.weight_offset == 0.0 and a.param("head_gate")
    assert (a.param("reads_cache"), b.param("reads_cache"), c.param("reads_cache")) == (False, True, False)
    assert c.position.kind == "rope_neox" and b.scale == 0.35
    assert [(r.layer, r.cache, r.writes_cache) for r in spec.run_order] == \
        [(0, 0, True), (1, 1, True), (2, 1, False), (3, 3, True), (4, 4, True)]
    ffs = [l.feed_forward for l in spec.layers]
    assert [f is None for f in ffs] == [False, True, False, True, False]
    assert ffs[0].param("groups") == (4, 2) and ffs[0].param("score_scale") == 1.5 and ffs[0].param("scores") == "softmax"
    assert ffs[2].param("groups") is None and ffs[2].param("score_scale") == 1.0
    names = expected_tensors(spec)
    for n in ("embed", "l0.norm1", "l0.norm2", "l0.mix.dq", "l0.mix.dq.norm", "l0.mix.uq", "l0.mix.dkv", "l0.mix.dkv.norm",
              "l0.mix.uk", "l0.mix.uv", "l0.mix.sink", "l0.mix.g", "l0.mix.o", "l0.mlp.router", "l0.mlp.e11.gate",
              "l0.mlp.e11.up", "l0.mlp.e0.down", "l1.mix.q.norm", "l1.mix.k.norm", "l1.mix.v", "l2.mix.q", "l2.mix.q.norm",
              "l2.mix.g", "final.norm", "head"):
        assert n in names, n
    for n in ("l1.norm2", "l1.mlp.router", "l2.mix.k", "l2.mix.v", "l2.mix.k.norm", "l1.mix.sink", "l0.mix.q", "embed.norm"):
        assert n not in names, n
    assert names["l0.mix.uq"][1].shape == (72, 40) and names["l0.mix.dkv"][1].shape == (32, 72)
    assert names["l0.mix.g"][1].shape == (72, 72) and names["l1.mix.g"][1].shape == (6, 72)
    assert names["l1.mix.v"][1].shape == (72, 72) and names["l1.mix.o"][1].shape == (72, 144)
    assert names["l0.mix.sink"][1].shape == (3,) and names["l0.mlp.e3.down"][1].shape == (72, 40)
    assert typed.to_dict()["layers"][2]["mixer"]["kv_from"] == 1


def test_cache_needs():
    """A layer that uses another's keys and values has no cache entry of its own."""
    import torch

    from reflex_b200.cache.specs import KVSpec
    from reflex_b200.engine.model import CausalLM

    _typed, spec = spec_of(pm.PID_B)
    specs = CausalLM(spec, torch.float32, "cpu").cache_entry_specs()
    assert specs == {0: KVSpec(1, 32, None),                      # the larger of 22 and 12 in steps of 16
                     1: KVSpec(1, 32, None, shared_kv=True),      # 18 + 4 in steps of 16 (of 64 in bfloat16)
                     3: KVSpec(3, 16, None)}
    _typed, spec = spec_of(pm.PID_E)
    assert sorted(CausalLM(spec, torch.bfloat16, "cpu").cache_entry_specs()) == [0, 1, 3]
    assert [r.cache for r in spec.run_order] == [0, 1, 0, 3, 3, 0]


def test_config_problems_are_named_together():
    from reflex_b200.errors import CheckpointError

    cfg = copy.deepcopy(pm.PID_A)
    del cfg["width"], cfg["postln_alpha"], cfg["embedding"]
    del cfg["layers"][0]["mixer"]["q_rank"]
    cfg["layers"][0]["mlp"]["router"]["groups"] = {"count": 4}
    del cfg["layers"][1]["mixer"]["rot"]["scaling"]["slow"]
    cfg["layers"][2]["mixer"]["kv_from"] = "1"
    del cfg["layers"][3]["mixer"]["rot"]["base"]
    cfg["layers"][4]["type"] = "delta"
    cfg["layers"][2]["mlp"] = {"kind": "dense"}
    with pytest.raises(CheckpointError) as e:
        spec_of(cfg)
    for part in ("width", "postln_alpha", "embedding.scale", "layers[0].mixer.q_rank", "layers[0].mlp.router.groups.keep",
                 "layers[1].mixer.rot.scaling.slow", "layers[2].mixer.kv_from", "layers[3].mixer.rot.base",
                 "layers[4].type='delta'", "layers[2].mlp.kind='dense'"):
        assert part in str(e.value), part

    def broken(change):
        cfg = copy.deepcopy(pm.PID_A)
        change(cfg["layers"])
        with pytest.raises(CheckpointError):
            spec_of(cfg)

    broken(lambda l: l[1]["mixer"].update(kv_heads=4))             # does not divide the heads
    broken(lambda l: l[1]["mixer"]["rot"].update(dims=18))         # more than the head has
    broken(lambda l: l[0]["mixer"]["rot"].update(dims=4))          # not the rotated part
    broken(lambda l: l[2]["mixer"].update(kv_from=2))              # itself
    broken(lambda l: l[2]["mixer"].update(kv_from=0))              # not an attention of this kind
    broken(lambda l: l[2]["mixer"].update(vdim=16))                # other values than the layer it reads
    broken(lambda l: l[4]["mixer"].update(kv_from=2))              # a layer without keys and values of its own
    broken(lambda l: l[0]["mlp"]["router"]["groups"].update(count=5))
    broken(lambda l: l[0]["mlp"]["router"]["groups"].update(keep=5))
    broken(lambda l: l[0]["mlp"]["router"].update(top=7))          # two groups of three hold six


def test_writer_and_loader_and_its_one_error(tmp_path):
    from reflex_b200.errors import CheckpointError
    from reflex_b200.weights import SafetensorsFile, write_random_model, write_safetensors
    from reflex_b200.weights.loader import Checkpoint, check_names_and_shapes

    d = write_random_model(pm.PID_A, 1, str(tmp_path / "m"), "bfloat16")
    cfg, w = pp.read_model(d)
    assert cfg["architecture"] == "Pidodra" and w["l0.mix.sink"].shape == (3,) and w["l0.mix.dkv"].shape == (32, 72)
    assert w["l0.norm1"].min() >= 0.89 and w["l1.mix.k.norm"].shape == (16,)
    _typed, spec = spec_of(cfg)
    ck = Checkpoint(d)
    check_names_and_shapes(spec, ck)
    ck.close()
    path = os.path.join(d, "model.safetensors")
    f = SafetensorsFile(path)
    tensors = {k: f.tensor(k).clone() for k in f.keys()}
    f.close()
    del tensors["l4.mix.g"]
    tensors["l2.mix.k"] = tensors["l1.mix.k"]
    tensors["l0.mix.uv"] = tensors["l0.mix.uv"][:, :23].contiguous()
    write_safetensors(path, list(tensors.items()))
    ck = Checkpoint(d)
    with pytest.raises(CheckpointError) as e:
        check_names_and_shapes(spec, ck)
    ck.close()
    assert "l4.mix.g" in str(e.value) and "l2.mix.k" in str(e.value) and "l0.mix.uv" in str(e.value)


# ------------------------------------------------- frequencies, order of rotated rows
@pytest.mark.parametrize("dims,base,sc", [(96, 10000.0, (6.0, 4096, 24.0, 1.5)), (8, 100.0, (4.0, 64, 8.0, 1.0)),
                                          (32, 1000.0, (16.0, 128, 4.0, 0.25)), (6, 30.0, (2.5, 40, 5.0, 0.5)),
                                          (16, 50.0, (3.0, 100000, 4.0, 2.0)), (10, 1e6, (1.0, 512, 32.0, 1.0)),
                                          (24, 500.0, (40.0, 8, 32.0, 16.0))])
def test_yarn_frequencies_and_magnitude(dims, base, sc):
    import torch

    from reflex_b200.config.spec import PositionSpec
    from reflex_b200.parts.registry import POSITIONS

    spec = PositionSpec("rope_yarn", dims, dims, base, tuple(zip(("factor", "original", "fast", "slow"), map(float, sc))))
    rot = POSITIONS.get(spec.kind)(spec, torch.float32, "cpu").rotation()
    ref = np.array(pp.yarn_frequencies(dims, base, *map(float, sc)))
    assert np.abs(1.0 / rot.denominators.double().numpy() / ref - 1.0).max() < 1e-6
    assert abs(rot.magnitude - pp.yarn_magnitude(sc[0])) < 1e-12 and rot.pairing == "half" and rot.rotary_dim == dims
    plain = np.array(pp.inverse_frequencies(dims, base))
    assert (ref <= plain * (1 + 1e-12)).all() and (ref >= plain / sc[0] * (1 - 1e-12)).all()


def test_yarn_keeps_fast_pairs_and_divides_slow_ones():
    f, g = pp.inverse_frequencies(96, 10000.0), pp.yarn_frequencies(96, 10000.0, 6.0, 4096, 24.0, 1.5)
    assert g[0] == f[0] and abs(g[47] * 6.0 - f[47]) < 1e-15   # about 650 turns, and a thirteenth of one
    assert any(f[i] / 6.0 * 1.01 < g[i] < f[i] * 0.99 for i in range(48))
    assert abs(pp.yarn_magnitude(math.e) - 1.1) < 1e-12 and pp.yarn_magnitude(1.0) == 1.0


def test_neighbouring_pairs_are_halves_in_another_order():
    """Rows of W_uq and W_dkv in the latent mixer's order turn as halves and give the
    same scores."""
    import torch

    from reflex_b200.config.spec import MixerSpec, PositionSpec
    from reflex_b200.parts.latent_attention import LatentAttention

    r, d = 8, 3
    part = LatentAttention(MixerSpec("latent_attention", hidden_size=8, num_heads=1, num_kv_heads=1, head_dim=d, v_head_dim=4,
                                     scale=1.0, position=PositionSpec("rope_neox", r, r, 100.0, (("pairing", "consecutive"),)),
                                     params=(("q_rank", 5), ("kv_rank", 6), ("rot_dim", r), ("eps", 1e-5))),
                           torch.float32, "cpu")
    order = part._pair_order()
    assert order["query"].tolist() == [0, 1, 2, 3, 5, 7, 9, 4, 6, 8, 10]
    assert order["key"].tolist() == [0, 1, 2, 3, 4, 5, 6, 8, 10, 12, 7, 9, 11, 13]
    assert part._rotation().pairing == "half"
    g = np.random.default_rng(0)
    q, k = g.standard_normal((1, 1, r)), g.standard_normal((1, 1, r))
    f, o = pp.inverse_frequencies(r, 100.0), (order["query"][d:] - d).numpy()
    a = (pp.rotate_neighbours(q, np.array([19]), f) * pp.rotate_neighbours(k, np.array([4]), f)).sum()
    b = (pp.rotate_halves(q[..., o], np.array([19]), f) * pp.rotate_halves(k[..., o], np.array([4]), f)).sum()
    assert abs(a - b) < 1e-12


# ------------------------------------------------------- the plain implementation
def test_rotations_of_halves_and_of_neighbours():
    t = np.zeros((3, 1, 8))
    t[:, 0, 1] = 1.0
    t[:, 0, 6] = 5.0   # beyond the rotated part
    f = pp.inverse_frequencies(4, 100.0)
    P = np.array([0, 1, 7])
    halves, pairs = pp.rotate_halves(t, P, f, 1.5), pp.rotate_neighbours(t, P, f)
    for r, p in enumerate(P):
        # halves: element 1 is the first of pair 1; neighbours: it is the second of pair 0
        assert abs(halves[r, 0, 1] - 1.5 * math.cos(p * 0.1)) < 1e-12 and abs(halves[r, 0, 3] - 1.5 * math.sin(p * 0.1)) < 1e-12
        assert abs(pairs[r, 0, 1] - math.cos(p)) < 1e-12 and abs(pairs[r, 0, 0] + math.sin(p)) < 1e-12
        assert halves[r, 0, 6] == pairs[r, 0, 6] == 5.0
    assert f == [1.0, 0.1]


def test_a_sink_joins_the_denominator_once():
    p = pp.softmax_rows(np.zeros((3, 3)), pp.causal(3), 0.0)
    assert np.allclose(p, [[1 / 2, 0, 0], [1 / 3, 1 / 3, 0], [1 / 4, 1 / 4, 1 / 4]])
    p = pp.softmax_rows(np.zeros((1, 1)), pp.causal(1), 50.0)
    assert 0 < p[0, 0] < 1e-20
    assert np.allclose(pp.softmax_rows(np.zeros((2, 2)), pp.causal(2), -90.0), [[1, 0], [0.5, 0.5]])


def test_experts_of_the_best_groups():
    s = np.array([0.05, 0.30, 0.01, 0.02, 0.25, 0.24, 0.03, 0.10])
    assert pp.choose_experts(s, 3, None) == [1, 4, 5]
    assert pp.choose_experts(s, 3, {"count": 4, "keep": 2}) == [1, 4, 5]
    assert pp.choose_experts(s, 4, {"count": 4, "keep": 2}) == [1, 4, 5, 0]     # not 7: its group is third
    assert pp.choose_experts(s, 3, {"count": 2, "keep": 1}) == [1, 0, 3]
    assert pp.choose_experts(s, 2, {"count": 8, "keep": 2}) == [1, 4]
    tie = np.full(6, 1 / 6)
    assert pp.choose_experts(tie, 3, {"count": 3, "keep": 2}) == [0, 1, 2]


def test_weights_are_the_scores_over_all_experts():
    """One expert chosen of two that are equal: half of its output times the factor."""
    W = 3
    w = {"router": np.zeros((2, W))}
    for e in range(2):
        w.update({f"e{e}.gate": np.ones((1, W)), f"e{e}.up": np.ones((1, W)), f"e{e}.down": np.ones((W, 1))})
    h = np.array([[1.0, 2.0, -1.0]])
    out = pp.experts_ff(h, w, {"router": {"experts": 2, "top": 1, "scale": 3.0}})
    assert np.allclose(out, 1.5 * 2.0 * pp.silu(2.0))


def test_norm_of_the_sum():
    """A mixer that gives nothing leaves the normed multiple of the stream: its own
    direction, whatever the factor."""
    cfg = pm.model(5, 4, 1e-12, 7.0, 1.0, [(pm.attention(1, 1, 2, 2, 1.0, (10.0, 2)), None)])
    w = {f"l0.mix.{n}": np.zeros(s) for n, s in (("q", (2, 4)), ("k", (2, 4)), ("v", (2, 4)), ("g", (1, 4)), ("o", (4, 2)))}
    w.update({"l0.mix.q.norm": np.ones(2), "l0.mix.k.norm": np.ones(2), "l0.norm1": np.array([1.0, 1.0, 2.0, 1.0])})
    x = np.array([[1.0, -2.0, 2.0, 4.0]])
    out = pp.layer_forward(x, cfg, w, 0, {})
    assert np.allclose(out, [[0.4, -0.8, 1.6, 1.6]])


# ------------------------------------------------- the test models show their mechanisms
def _logits(name, cfg_change=None, weight_change=None, n=80):
    cfg, w = pp.read_model(pm.model_folder(name))
    cfg, w = copy.deepcopy(cfg), dict(w)
    if cfg_change:
        cfg_change([l["mixer"] for l in cfg["layers"]], cfg)
    if weight_change:
        weight_change(w)
    return pp.forward(cfg, w, pm.tokens(n, cfg["vocab"], 11))


def _moved(a, b):
    return np.abs(a - b).max() / np.abs(a).max()


def test_the_test_models_show_every_mechanism():
    base = _logits("A")

    def scaled(name, f=0.0, o=0.0):
        def change(w):
            w[name] = w[name] * f + o
        return change

    def router(i, **kw):
        return lambda m, c: c["layers"][i]["mlp"]["router"].update(**kw)

    changes = {
        "alpha": dict(cfg_change=lambda m, c: c.update(postln_alpha=1.4)),
        "embedding scale": dict(cfg_change=lambda m, c: c["embedding"].update(scale=2.0)),
        "eps": dict(cfg_change=lambda m, c: c["norm"].update(eps=1e-2)),
        "latent scale": dict(cfg_change=lambda m, c: m[0].update(scale=0.62)),
        "latent base": dict(cfg_change=lambda m, c: m[0]["rot"].update(base=900.0)),
        "sink": dict(weight_change=scaled("l0.mix.sink", 1.0, -30.0)),
        "element gate": dict(weight_change=scaled("l0.mix.g")),
        "query latent norm": dict(weight_change=lambda w: w.update({"l0.mix.dq.norm": np.ones(40)})),
        "latent norm": dict(weight_change=lambda w: w.update({"l0.mix.dkv.norm": np.ones(24)})),
        "rotated dims": dict(cfg_change=lambda m, c: [m[i]["rot"].update(dims=16) for i in (1, 2)]),
        "factor": dict(cfg_change=lambda m, c: [m[i]["rot"]["scaling"].update(factor=4.5) for i in (1, 2)]),
        "original": dict(cfg_change=lambda m, c: [m[i]["rot"]["scaling"].update(original=400) for i in (1, 2)]),
        "slow": dict(cfg_change=lambda m, c: [m[i]["rot"]["scaling"].update(slow=4.0) for i in (1, 2)]),
        "scale": dict(cfg_change=lambda m, c: m[2].update(scale=0.4)),
        "query norm": dict(weight_change=lambda w: w.update({"l2.mix.q.norm": np.ones(16)})),
        "key norm": dict(weight_change=lambda w: w.update({"l1.mix.k.norm": np.ones(16)})),
        "head gate": dict(weight_change=scaled("l2.mix.g")),
        "own values": dict(weight_change=scaled("l1.mix.v", 0.9)),
        "groups": dict(cfg_change=router(0, groups=None)),
        "kept groups": dict(cfg_change=router(4, groups={"count": 3, "keep": 3})),
        "router scale": dict(cfg_change=router(0, scale=1.0)),
        "experts chosen": dict(cfg_change=router(2, top=1)),
        "norm on the mixer's sum": dict(weight_change=lambda w: w.update({"l3.norm1": np.ones(72)})),
        "norm on the feed-forward's sum": dict(weight_change=lambda w: w.update({"l0.norm2": np.ones(72)})),
        "final norm": dict(weight_change=lambda w: w.update({"final.norm": np.ones(72)})),
    }
    for what, kw in changes.items():
        assert _moved(base, _logits("A", **kw)) > 2e-3, what  # ten times the 32-bit tests' tolerance
