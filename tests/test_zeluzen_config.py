"""The Zeluzen configuration class and the plain implementation's own pieces, on the CPU.

What config.json says must arrive in the ModelSpec unchanged (sizes, constants, layer order), the tensors the model
declares must be the file's names and shapes, and a configuration that cannot be built is refused in words.  The plain
implementation's mechanisms are checked against second, independent formulations of the same equations.
"""
import cmath
import math

import numpy as np
import pytest
import plain_zeluzen as pz

from inferllm_b200 import ConfigError, ZeluzenConfig, config_from_dict
from inferllm_b200.cache import cache_requests
from inferllm_b200.weights import tensor_decls

S, A = "wkv", "attention"


def f64(w):
    return {k: np.asarray(v, np.float64) for k, v in w.items()}


def sample_config():
    return pz.make_config([(S, pz.wkv_mixer(heads=5, dim=10), None),
                           (A, pz.attn_mixer(heads=6, kv_heads=3, dim=12, vdim=18, size=31, scale=0.37, base=777.0, dims=8, scaling=(2.5, 1.5, 3.5, 96)),
                            pz.dense_mlp(52)),
                           (S, pz.wkv_mixer(heads=2, dim=24), pz.moe_mlp(ff=20, experts=7, identity=3, top=4)),
                           (A, pz.attn_mixer(heads=3, kv_heads=3, dim=12, vdim=18, size=45, scale=0.2, base=777.0, dims=8, scaling=(2.5, 1.5, 3.5, 96), kv_from=1),
                            pz.moe_mlp(ff=16, experts=4, identity=0, top=2)),
                           (A, pz.attn_mixer(heads=2, kv_heads=1, size=0, scaling=None), None)],
                          width=56, vocab=77, eps=3e-5)


def test_spec_carries_every_size_and_constant():
    spec = config_from_dict(sample_config()).model_spec()
    assert (spec.hidden_size, spec.vocab_size) == (56, 77)
    assert [(e.layer, e.cache, e.writes, e.reenter) for e in spec.schedule] == \
        [(0, 0, True, False), (1, 1, True, False), (2, 2, True, False), (3, 1, False, False), (4, 4, True, False)]
    assert [l.block for l in spec.layers] == ["outnorm_mixer", "outnorm", "outnorm", "outnorm", "outnorm_mixer"]
    for l in spec.layers:
        assert sorted(l.norms) == (["norm1", "norm2"] if l.block == "outnorm" else ["norm1"])
        assert all(n.kind == "rmsnorm" and n["eps"] == 3e-5 and n["size"] == 56 for n in l.norms.values())
    s, a, s2, reader, plain = (l.mixer for l in spec.layers)
    assert s.kind == "wkv" and (s["n_heads"], s["head_dim"], s["norm_eps"]) == (5, 10, 3e-5)
    assert (s2["n_heads"], s2["head_dim"]) == (2, 24)
    assert a.kind == "attention" and (a["n_heads"], a["n_kv_heads"], a["head_dim"], a["v_head_dim"], a["chunk"], a["scale"]) == (6, 3, 12, 18, 31, 0.37)
    assert a["unit_sink"] is True and a["qk_norm"] == "head" and "own_kv" not in a.params
    pos = a["position"]
    assert pos.kind == "rope_pairs" and (pos["theta"], pos["rot_dim"], pos["head_dim"]) == (777.0, 8, 12)
    assert pos["scaling"] == {"factor": 2.5, "original": 96.0, "low": 1.5, "high": 3.5}
    assert reader["own_kv"] is False and (reader["n_heads"], reader["chunk"], reader["scale"]) == (3, 45, 0.2)
    assert plain["chunk"] == 0 and "scaling" not in plain["position"].params
    f = spec.layers[1].ffn
    assert f.kind == "gated_mlp" and (f["intermediate_size"], f["activation"]) == (52, "silu")
    f = spec.layers[2].ffn
    assert f.kind == "routed_mlp" and (f["intermediate_size"], f["experts"], f["identity_experts"], f["top"]) == (20, 7, 3, 4)
    assert (f["expert_kind"], f["activation"], f["scoring"], f["choice_correction"], f["renormalize"]) == ("plain", "relu_squared", "softmax_all", True, False)
    assert spec.layers[3].ffn["identity_experts"] == 0 and spec.layers[0].ffn.kind == ""
    assert spec.embedding["norm"]["eps"] == 3e-5 and spec.head["tied"] is False


def test_the_python_face_is_typed_and_round_trips():
    c = config_from_dict(sample_config())
    assert isinstance(c, ZeluzenConfig) and c.architecture == "Zeluzen"
    assert ZeluzenConfig.from_dict(c.to_dict()) == c and c.to_dict()["width"] == 56


def test_declared_tensors_are_the_files_names_and_shapes():
    cfg = sample_config()
    decls = {name: tuple(shape) for name, (shape, _) in tensor_decls(config_from_dict(cfg)).items()}
    want = {k: tuple(v[0]) for k, v in pz.tensor_shapes(cfg).items()}
    for i in (0, 2):      # the inner size of the decay's map is whatever the file has
        n = cfg["layers"][i]["mixer"]["heads"] * cfg["layers"][i]["mixer"]["dim"]
        want["l%d.mix.w1" % i], want["l%d.mix.w2" % i] = (-1, 56), (n, -1)
    assert decls == want
    named = sample_config()
    for i in (0, 2):
        named["layers"][i]["mixer"]["decay_rank"] = 9
    decls = {name: tuple(shape) for name, (shape, _) in tensor_decls(config_from_dict(named)).items()}
    assert decls == {k: tuple(v[0]) for k, v in pz.tensor_shapes(cfg, rank=9).items()}


@pytest.mark.parametrize("edit, word", [
    (lambda c: c["layers"][0].__setitem__("type", "convolution"), "unknown type"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("heads", 0), "heads and dim"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("kv_heads", 4), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"]["mask"].__setitem__("size", 0), "mask.size"),
    (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 5), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 14), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("low"), "low"),
    (lambda c: c["layers"][3]["mixer"].__setitem__("kv_from", 2), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].__setitem__("kv_from", 4), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].__setitem__("vdim", 20), "kv_from"),
    (lambda c: c["layers"][1]["mlp"].__setitem__("kind", "sparse"), "kind"),
    (lambda c: c["layers"][2]["mlp"]["router"].__setitem__("top", 11), "top"),
    (lambda c: c["layers"][2]["mlp"].pop("expert"), "expert"),
    (lambda c: c["norm"].__setitem__("eps", 0.0), "eps"),
    (lambda c: c.__setitem__("layers", []), "layers"),
])
def test_what_cannot_be_built_is_refused_in_words(edit, word):
    cfg = sample_config()
    edit(cfg)
    with pytest.raises(ConfigError) as e:
        tensor_decls(config_from_dict(cfg))
    assert word in str(e.value)


@pytest.mark.parametrize("own, readers, want", [
    (31, [31], (None, 31)),            # the same mask: the pages of a finished chunk go back at once
    (31, [45], (45, None)),            # another chunk: whatever either of them may still see
    (45, [31], (45, None)),
    (31, [0], (None, None)),           # a reader that sees all earlier positions
    (0, [31], (None, None)),
    (20, [50, 7], (50, None)),
])
def test_a_shared_cache_entry_keeps_what_its_readers_see(own, readers, want):
    cfg = pz.make_config([(A, pz.attn_mixer(size=own), None)] + [(A, pz.attn_mixer(size=n, kv_from=0), None) for n in readers])
    got = cache_requests(config_from_dict(cfg))
    assert list(got) == [0] and (got[0].get("window"), got[0].get("chunk")) == want


# ---------------------------------------------------------------- the plain implementation against second formulations


def test_recurrence_against_its_unrolled_form():
    """o_t = sum over s < t of (r_t . (k_s * product of the decays between them)) v_s, plus the bonus term."""
    rng = np.random.default_rng(0)
    n, H, d, dv = 9, 2, 5, 4
    r, k = rng.standard_normal((2, n, H, d))
    v, w, u = rng.standard_normal((n, H, dv)), rng.uniform(0.2, 1.0, (n, H, d)), rng.standard_normal((H, d))
    got = pz.wkv_scan(r, k, v, w, u)
    for a in range(H):
        for t in range(n):
            o = (r[t, a] * u[a] * k[t, a]).sum() * v[t, a]
            for s in range(t):
                o = o + (r[t, a] * k[s, a] * w[s + 1:t, a].prod(0)).sum() * v[s, a]
            assert np.allclose(got[t, a], o, rtol=1e-10, atol=1e-12)


def test_blend_and_decay_by_hand():
    x = np.array([[1.0, 2.0], [3.0, 4.0], [5.0, 7.0]])
    assert np.allclose(pz.blend(x, np.array([0.0, 1.0])), [[1, 0], [3, 2], [5, 4]])
    assert np.allclose(pz.blend(x, np.array([0.25, 0.5])), [[0.75, 1.0], [2.5, 3.0], [4.5, 5.5]])
    w1, w2, w0 = np.array([[0.5, 0.0]]), np.array([[2.0], [0.0]]), np.array([0.0, -1.0])
    w = pz.channel_decay(x, w1, w2, w0)
    assert math.isclose(w[1, 0], math.exp(-math.exp(2.0 * math.tanh(1.5)))) and math.isclose(w[1, 1], math.exp(-math.exp(-1.0)))


def test_attention_against_masked_matrices():
    cfg = pz.make_config([(A, pz.attn_mixer(heads=4, kv_heads=2, dim=8, vdim=6, size=7, dims=4), None)], width=20)
    m = cfg["layers"][0]["mixer"]
    W = f64(pz.random_weights(cfg, 3))
    x = np.random.default_rng(1).standard_normal((23, 20))
    k, v = pz.keys_and_values(x, W, "l0.mix.", m, 1e-5)
    got = pz.attend(x, W, "l0.mix.", m, 1e-5, (k, v))
    q = (x @ W["l0.mix.q"].T).reshape(23, 4, 8)
    q = q / np.sqrt((q ** 2).mean(-1, keepdims=True) + 1e-5) * W["l0.mix.q.norm"]
    q = np.stack([pz.rotate_pairs(q[t], t, m["rot"]) for t in range(23)])
    i, j = np.arange(23)[:, None], np.arange(23)[None, :]
    mask = (j <= i) & (i // 7 == j // 7)
    out = []
    for a in range(4):
        e = np.where(mask, np.exp(q[:, a] @ k[:, a // 2].T * m["scale"]), 0.0)
        out.append(e / (1.0 + e.sum(-1, keepdims=True)) @ v[:, a // 2])
    assert np.allclose(got, np.concatenate(out, -1) @ W["l0.mix.o"].T)


def test_rotation_as_complex_numbers_and_its_frequencies_by_hand():
    x = np.random.default_rng(2).standard_normal(10)
    rot = {"base": 50.0, "dims": 6}
    y = pz.rotate_pairs(x, 13, rot)
    for i in range(3):
        z = complex(x[2 * i], x[2 * i + 1]) * cmath.exp(1j * 13 * 50.0 ** (-i / 3))
        assert cmath.isclose(z, complex(y[2 * i], y[2 * i + 1]))
    assert np.array_equal(y[6:], x[6:])
    # wavelengths 2 pi 10^i against an original length of 200: shorter than 200 / 4, between, longer than 200 / 1
    f = pz.frequencies({"base": 1e4, "dims": 8, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 200}})
    assert f[0] == 1.0
    s = (200 / (2 * math.pi * 10) - 1.0) / 3.0
    assert math.isclose(f[1], (1 - s) * 0.1 / 8 + s * 0.1)
    assert math.isclose(f[2], 0.01 / 8) and math.isclose(f[3], 0.001 / 8)


def test_routing_by_hand():
    """The correction decides the choice and leaves the weights alone; identity experts give their input back."""
    W = {"m.router": np.log(np.array([[4.0], [3.0], [2.0], [1.0]])), "m.correction": np.array([0.0, -1.0, 0.0, 0.5]),
         "m.e0.up": np.array([[2.0], [-1.0]]), "m.e0.down": np.array([[1.0, 7.0]]), "m.e1.up": np.ones((2, 1)), "m.e1.down": np.ones((1, 2))}
    y = pz.routed(np.array([[1.0]]), W, "m.", {"expert": {"ff": 2}, "router": {"experts": 2, "identity": 2, "top": 2}})
    # scores 0.4, 0.3, 0.2, 0.1: chosen by 0.6 (the last, an identity expert) and 0.4 (the first)
    assert np.allclose(y, [[0.1 * 1.0 + 0.4 * 4.0]])


def test_whole_model_is_causal():
    cfg = sample_config()
    W = f64(pz.random_weights(cfg, 5))
    ids = np.random.default_rng(3).integers(0, 77, 40).tolist()
    a = pz.forward(cfg, W, ids)
    b = pz.forward(cfg, W, ids[:30] + [1] * 10)
    assert np.allclose(a[:30], b[:30]) and not np.allclose(a[30:], b[30:])
