"""Zivulix without a GPU: configuration, the model description built from it
(cache needs, tensor names, which layers mix values), the random-weights writer
and the loader's one error; the plain implementation against closed forms; and
that the test models' weights make every mechanism show."""

import copy
import math
import os

import numpy as np
import pytest

import plain_zivulix as pz
import zivulix_models as zm


def spec_of(cfg):
    from reflex_b200 import models  # noqa: F401
    from reflex_b200.config.registry import spec_from_config_dict

    return spec_from_config_dict(cfg)


def test_config_to_model_description():
    from reflex_b200.engine.model import expected_tensors

    typed, spec = spec_of(zm.ZIV_A)
    assert spec.architecture == "zivulix" and (spec.vocab_size, spec.hidden_size) == (97, 72)
    assert not spec.tie_word_embeddings and spec.embedding_norm_name == "embed.norm"
    assert spec.embedding_norm.weight_offset == spec.final_norm.weight_offset == 1.0
    assert [l.block for l in spec.layers] == ["postnorm"] * 5
    assert [l.mixer.kind for l in spec.layers] == ["gated_delta", "capped_attention", "latent_attention",
                                                   "capped_attention", "gated_delta"]
    assert [None if l.feed_forward is None else (l.feed_forward.kind, l.feed_forward.intermediate_size)
            for l in spec.layers] == [("geglu", 96), None, ("geglu", 80), ("geglu", 48), None]
    d, a, lat, a2 = (l.mixer for l in spec.layers[:4])
    assert (d.num_heads, d.num_kv_heads, d.head_dim, d.value_dim, d.param("taps")) == (4, 2, 16, 24, 4)
    assert abs(d.scale - 0.25) < 1e-15 and d.param("unit_eps") == 1e-6 and d.param("eps") == 1e-5
    assert (a.num_heads, a.num_kv_heads, a.head_dim, a.value_dim, a.window, a.scale) == (6, 3, 16, 24, 20, 0.8)
    assert a.param("softcap") == 5.0 and a.param("unit_eps") == 1e-5 and a.param("bias")
    assert a.position.kind == "rope_linear" and (a.position.rotary_dim, a.position.theta) == (8, 100.0)
    assert dict(a.position.params)["factor"] == 2.0
    assert (a.param("value_mix"), a2.param("value_mix")) == ("first", "mix")
    assert (lat.num_heads, lat.head_dim, lat.value_dim, lat.param("rot_dim"), lat.param("kv_rank"), lat.window) == \
        (3, 16, 24, 8, 40, None)
    assert lat.position.rotary_dim == 8 and dict(lat.position.params)["factor"] == 1.0
    names = expected_tensors(spec)
    for n in ("embed", "embed.norm", "l0.norm1", "l0.norm2", "l0.mix.q.conv", "l0.mix.b", "l0.mix.a", "l0.mix.A_log",
              "l0.mix.dt_bias", "l0.mix.g", "l0.mix.norm", "l0.mlp.down", "l1.norm1", "l1.mix.q.b", "l1.mix.vmix",
              "l3.mix.vmix", "l2.mix.dkv", "l2.mix.dkv.norm", "l2.mix.uk", "l2.mix.uv", "final.norm", "head"):
        assert n in names, n
    for n in ("l1.norm2", "l1.mlp.up", "l4.norm2", "l2.mix.k", "l2.mix.dq", "l0.mix.q.b", "l1.mix.o.b"):
        assert n not in names, n
    assert names["l0.mix.v"][1].shape == (96, 72) and names["l0.mix.k"][1].shape == (32, 72)
    assert names["l0.mix.v.conv"][1].shape == (96, 4) and names["l0.mix.norm"][1].shape == (24,)
    assert names["l1.mix.v"][1].shape == (72, 72) and names["l1.mix.vmix"][1].shape == ()
    assert names["l2.mix.q"][1].shape == (72, 72) and names["l2.mix.dkv"][1].shape == (48, 72)
    assert names["l2.mix.uk"][1].shape == (48, 40) and names["l2.mix.o"][1].shape == (72, 72)
    assert typed.to_dict()["layers"][1]["mixer"]["rot"]["scaling"]["factor"] == 2.0


def test_cache_needs_and_which_layers_mix_values():
    import torch

    from reflex_b200.cache.specs import KVSpec, StateSpec
    from reflex_b200.engine.model import CausalLM, expected_tensors

    _typed, spec = spec_of(zm.ZIV_B)
    specs = CausalLM(spec, torch.float32, "cpu").cache_entry_specs()
    assert specs[0] == KVSpec(1, 32, None, shared_kv=True)          # 18 + 4 in steps of 16 (of 64 in bfloat16)
    assert specs[1] == StateSpec((2 * 7 * 12,), "float32")           # one tap: no filter state; 10 channels in fours
    assert specs[2] == KVSpec(1, 32, None)                           # the larger of 22 and 12 in steps of 16
    assert specs[3] == StateSpec((232 + 50 * 36,), "float32")        # 2 * 116 filter inputs, then S
    assert spec.layers[2].mixer.param("value_mix") is None and "l2.mix.vmix" not in expected_tensors(spec)
    assert dict(spec.layers[2].mixer.position.params)["factor"] == 1.0
    _typed, spec = spec_of(zm.ZIV_E)
    assert [l.mixer.param("value_mix") for l in spec.layers if l.mixer.kind == "capped_attention"] == \
        [None, "first", "mix", "mix"]
    assert [l.mixer.window for l in spec.layers if l.mixer.kind == "capped_attention"] == [200, 130, 65, 1]


def test_config_problems_are_named_together():
    from reflex_b200.errors import CheckpointError

    cfg = copy.deepcopy(zm.ZIV_A)
    del cfg["width"]
    del cfg["layers"][0]["mixer"]["conv"]
    cfg["layers"][1]["mixer"]["mask"] = {}
    cfg["layers"][1]["mixer"]["rot"]["scaling"] = {"factor": "2"}
    del cfg["layers"][2]["mixer"]["rot"]["base"]
    cfg["layers"][3]["mixer"]["kv_heads"] = None
    cfg["layers"][4]["type"] = "retention"
    cfg["layers"][0]["mlp"] = {"kind": "moe"}
    with pytest.raises(CheckpointError) as e:
        spec_of(cfg)
    for part in ("width", "layers[0].mixer.conv", "layers[1].mixer.mask.size", "layers[1].mixer.rot.scaling.factor",
                 "layers[2].mixer.rot.base", "layers[3].mixer.kv_heads", "layers[4].type='retention'",
                 "layers[0].mlp.kind='moe'"):
        assert part in str(e.value), part

    def broken(change):
        cfg = copy.deepcopy(zm.ZIV_A)
        change(cfg["layers"])
        with pytest.raises(CheckpointError):
            spec_of(cfg)

    broken(lambda l: l[0]["mixer"].update(kv_heads=3))            # does not divide the heads
    broken(lambda l: l[1]["mixer"]["rot"].update(dims=18))        # more than the head has
    broken(lambda l: l[2]["mixer"]["rot"].update(dims=4))         # not the rotated part
    broken(lambda l: l[3]["mixer"].update(vdim=20))               # mixed values of another width
    broken(lambda l: l[1]["mixer"].update(softcap=-1.0))


def test_writer_and_loader_and_its_one_error(tmp_path):
    from reflex_b200.errors import CheckpointError
    from reflex_b200.weights import SafetensorsFile, write_random_model, write_safetensors
    from reflex_b200.weights.loader import Checkpoint, check_names_and_shapes

    d = write_random_model(zm.ZIV_A, 1, str(tmp_path / "m"), "bfloat16")
    cfg, w = pz.read_model(d)
    assert cfg["architecture"] == "Zivulix" and w["l1.mix.vmix"].shape == () and w["l2.mix.dkv"].shape == (48, 72)
    assert np.abs(w["l0.norm1"]).max() <= 0.11 and w["l0.mix.norm"].min() >= 0.89
    _typed, spec = spec_of(cfg)
    ck = Checkpoint(d)
    check_names_and_shapes(spec, ck)
    ck.close()
    path = os.path.join(d, "model.safetensors")
    f = SafetensorsFile(path)
    tensors = {k: f.tensor(k).clone() for k in f.keys()}
    f.close()
    del tensors["l4.mix.A_log"]
    tensors["l0.mix.q.b"] = tensors["l0.norm1"]
    tensors["l2.mix.uv"] = tensors["l2.mix.uv"][:, :39].contiguous()
    write_safetensors(path, list(tensors.items()))
    ck = Checkpoint(d)
    with pytest.raises(CheckpointError) as e:
        check_names_and_shapes(spec, ck)
    ck.close()
    assert "l4.mix.A_log" in str(e.value) and "l0.mix.q.b" in str(e.value) and "l2.mix.uv" in str(e.value)


# ------------------------------------------------------- the plain implementation
def test_rotation_divides_frequencies_and_keeps_scores_to_the_distance():
    t = np.zeros((3, 1, 8))
    t[:, 0, 1] = 1.0   # pairs with dimension 3 when four dimensions turn
    t[:, 0, 6] = 5.0   # beyond the rotated part
    out = pz.rotate(t, np.array([0, 1, 7]), 4, 100.0, 5.0)
    f1 = 100.0 ** (-2.0 / 4) / 5.0
    for r, p in enumerate([0, 1, 7]):
        assert abs(out[r, 0, 1] - math.cos(p * f1)) < 1e-12 and abs(out[r, 0, 3] - math.sin(p * f1)) < 1e-12
        assert out[r, 0, 6] == 5.0 and out[r, 0, 0] == 0.0
    g = np.random.default_rng(0)
    q, k = g.standard_normal((1, 1, 8)), g.standard_normal((1, 1, 8))
    a = (pz.rotate(q, np.array([9]), 8, 50.0) * pz.rotate(k, np.array([4]), 8, 50.0)).sum()
    b = (pz.rotate(q, np.array([105]), 8, 50.0) * pz.rotate(k, np.array([100]), 8, 50.0)).sum()
    assert abs(a - b) < 1e-9


def test_window_and_softmax():
    m = pz.visible(6, 3)
    assert m[5].tolist() == [False, False, False, True, True, True] and m[1].tolist() == [True, True] + [False] * 4
    assert pz.visible(4, None)[3].all() and not pz.visible(4, None)[0, 1]
    p = pz.softmax_rows(np.zeros((6, 6)), m)
    assert np.allclose(p[5], [0, 0, 0, 1 / 3, 1 / 3, 1 / 3]) and np.allclose(p[0], [1, 0, 0, 0, 0, 0])


def test_values_are_mixed_with_the_first_layers_own():
    carry, w = {}, {"vmix": np.array(0.25)}
    v1, v2 = np.full((2, 1, 3), 4.0), np.full((2, 1, 3), 8.0)
    assert pz.mixed_values(v2, {"v_mix": False}, {}, carry) is v2 and not carry
    assert pz.mixed_values(v1, {"v_mix": True}, w, carry) is v1
    assert np.allclose(pz.mixed_values(v2, {"v_mix": True}, w, carry), 7.0)
    assert np.allclose(pz.mixed_values(v2, {"v_mix": True}, w, carry), 7.0)   # with the first, not the last


def test_capped_scores_of_unit_queries_and_keys():
    """One head whose query and key are the same direction: the raw score is
    dim * scale, whatever the length of the projections."""
    m = {"heads": 1, "kv_heads": 1, "dim": 4, "vdim": 1, "scale": 2.0, "softcap": 3.0, "rot": {"base": 10.0, "dims": 2}}
    W = 3
    w = {"q": np.zeros((4, W)), "k": np.zeros((4, W)), "v": np.array([[0.0, 1.0, 0.0]]), "o": np.array([[1.0]]),
         "q.b": np.array([0.0, 0.0, 5.0, 0.0]), "k.b": np.zeros(4), "v.b": np.zeros(1)}
    w["k"][2, 0] = 7.0   # the token with h[0] > 0 has a key along dimension 2, the other none
    h = np.array([[1.0, 10.0, 0.0], [0.0, 20.0, 0.0]])
    out = pz.attention(h, w, m, 1e-12, {})
    s = 3.0 * np.tanh(2.0 * 4 / 3.0)
    assert abs(out[0, 0] - 10.0) < 1e-9
    assert abs(out[1, 0] - (10.0 * np.exp(s) + 20.0) / (np.exp(s) + 1.0)) < 1e-5


def test_latent_attention_shares_one_rotated_key_part():
    """With no unrotated part in the queries, the scores come from the shared part alone,
    and so are the same for every head with the same rotated query."""
    g = np.random.default_rng(1)
    T, W, H, d, r, dv, kr = 5, 6, 2, 3, 4, 2, 5
    m = {"heads": H, "dim": d, "rot_dim": r, "vdim": dv, "kv_rank": kr, "scale": 0.7, "rot": {"base": 20.0, "dims": r}}
    qr = g.standard_normal((r, W))
    q = np.concatenate([np.zeros((d, W)), qr, np.zeros((d, W)), qr])
    w = {"q": q, "dkv": g.standard_normal((kr + r, W)), "dkv.norm": g.random(kr) + 0.5,
         "uk": g.standard_normal((H * d, kr)), "uv": g.standard_normal((H * dv, kr)), "o": np.eye(H * dv)}
    h = g.standard_normal((T, W))
    out = pz.latent_attention(h, w, m, 1e-6)
    down = h @ w["dkv"].T
    c = pz.rms_unit(down[:, :kr], 1e-6) * w["dkv.norm"]
    pos = np.arange(T)
    kk = pz.rotate(down[:, None, kr:], pos, r, 20.0)[:, 0]
    qq = pz.rotate((h @ qr.T)[:, None], pos, r, 20.0)[:, 0]
    p = pz.softmax_rows(qq @ kk.T * 0.7, pz.visible(T, None))
    assert np.allclose(out, p @ (c @ w["uv"].T))


def test_gated_delta_rule_decays_then_writes_then_reads():
    d, dv = 3, 2
    g = np.random.default_rng(3)
    k = pz.unit(g.standard_normal((1, 1, d)))[0, 0]
    v1, v2, q = g.standard_normal(dv), g.standard_normal(dv), g.standard_normal(d)
    ks, qs = np.stack([k, k])[:, None], np.stack([q, q])[:, None]
    vs = np.stack([v1, v2])[:, None]
    # a write rate of one along the same unit key replaces what was there, whatever the decay
    o = pz.gated_delta_scan(qs, ks, vs, np.array([[0.9], [0.5]]), np.ones((2, 1)))
    assert np.allclose(o[0, 0], v1 * (k @ q), atol=1e-5) and np.allclose(o[1, 0], v2 * (k @ q), atol=1e-5)
    # a write rate of zero only decays
    o = pz.gated_delta_scan(qs, ks, vs, np.array([[0.9], [0.5]]), np.array([[1.0], [0.0]]))
    assert np.allclose(o[1, 0], 0.5 * v1 * (k @ q), atol=1e-5)
    # half a write of the difference from the decayed memory
    o = pz.gated_delta_scan(qs, ks, vs, np.array([[1.0], [0.5]]), np.array([[1.0], [0.25]]))
    assert np.allclose(o[1, 0], (0.5 * v1 + 0.25 * (v2 - 0.5 * v1)) * (k @ q), atol=1e-5)


def test_causal_convolution_looks_back_and_starts_from_zeros():
    x = np.arange(1.0, 6.0)[:, None]
    out = pz.causal_conv(x, np.array([[100.0, 10.0, 1.0]]))
    assert out[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0, 345.0]


def test_gelu_and_the_norm_around_zero():
    z = np.array([-3.0, 0.0, 1.0])
    assert np.allclose(pz.gelu_tanh(z), [-0.00363739, 0.0, 0.84119199], atol=1e-7)
    x = np.array([[3.0, 4.0]])
    assert np.allclose(pz.norm_around_zero(x, np.array([0.0, 1.0]), 0.0), [[3 / math.sqrt(12.5), 8 / math.sqrt(12.5)]])


# ------------------------------------------------- the test models show their mechanisms
def _logits(name, cfg_change=None, weight_change=None, n=90):
    cfg, w = pz.read_model(zm.model_folder(name))
    cfg, w = copy.deepcopy(cfg), dict(w)
    if cfg_change:
        cfg_change([l["mixer"] for l in cfg["layers"]], cfg)
    if weight_change:
        weight_change(w)
    return pz.forward(cfg, w, zm.tokens(n, cfg["vocab"], 11))


def _moved(a, b):
    return np.abs(a - b).max() / np.abs(a).max()


def test_the_test_models_show_every_mechanism():
    base = _logits("A")

    def scaled(name, f=0.0, o=0.0):
        def change(w):
            w[name] = w[name] * f + o
        return change

    def first_tap(w):
        w["l0.mix.v.conv"] = w["l0.mix.v.conv"].copy()
        w["l0.mix.v.conv"][:, 0] = 0.0

    changes = {
        "window": dict(cfg_change=lambda m, c: m[1]["mask"].update(size=21)),
        "second window": dict(cfg_change=lambda m, c: m[3]["mask"].update(size=32)),
        "rotated dims": dict(cfg_change=lambda m, c: m[1]["rot"].update(dims=16)),
        "divided frequencies": dict(cfg_change=lambda m, c: m[1]["rot"]["scaling"].update(factor=2.5)),
        "base": dict(cfg_change=lambda m, c: m[2]["rot"].update(base=900.0)),
        "cap": dict(cfg_change=lambda m, c: m[1].update(softcap=500.0)),
        "scale": dict(cfg_change=lambda m, c: m[2].update(scale=0.62)),
        "no mix": dict(cfg_change=lambda m, c: m[3].update(v_mix=False)),
        "eps": dict(cfg_change=lambda m, c: c["norm"].update(eps=1e-2)),
        "mix": dict(weight_change=scaled("l3.mix.vmix", 1.0, 0.2)),
        "query bias": dict(weight_change=scaled("l1.mix.q.b")),
        "value bias": dict(weight_change=scaled("l1.mix.v.b")),
        "oldest tap": dict(weight_change=first_tap),
        "decay": dict(weight_change=scaled("l0.mix.A_log", 1.0, 0.5)),
        "step bias": dict(weight_change=scaled("l0.mix.dt_bias", 1.0, 0.5)),
        "write rate": dict(weight_change=scaled("l0.mix.b")),
        "gate": dict(weight_change=scaled("l0.mix.g")),
        "delta norm": dict(weight_change=lambda w: w.update({"l0.mix.norm": np.ones(24)})),
        "latent norm": dict(weight_change=lambda w: w.update({"l2.mix.dkv.norm": np.ones(40)})),
        "embedding norm": dict(weight_change=scaled("embed.norm")),
        "norm on the mixer": dict(weight_change=scaled("l2.norm1")),
        "norm on the feed-forward": dict(weight_change=scaled("l0.norm2")),
        "final norm": dict(weight_change=scaled("final.norm")),
    }
    for what, kw in changes.items():
        assert _moved(base, _logits("A", **kw)) > 2e-3, what  # ten times the 32-bit tests' tolerance
    # the first mixing layer's own number is not used
    assert _moved(base, _logits("A", weight_change=scaled("l1.mix.vmix", 1.0, 0.3))) == 0.0
