"""The Fifotar configuration class and the plain implementation's own pieces, on the CPU.

What config.json says must arrive in the ModelSpec unchanged (sizes, constants, layer order), the tensors the model
declares must be the file's names and shapes, and a configuration that cannot be built is refused in words.  The plain
implementation's mechanisms are checked against second, independent formulations of the same equations.
"""
import cmath
import math

import numpy as np
import pytest
import plain_fifotar as pf

from inferllm_b200 import ConfigError, FifotarConfig, config_from_dict
from inferllm_b200.weights import tensor_decls

S, A, L = "delta", "attention", "latent_attention"


def f64(w):
    return {k: np.asarray(v, np.float64) for k, v in w.items()}


def sample_config():
    return pf.make_config([(S, pf.delta_mixer(heads=6, kv_heads=3, dim=10, vdim=14, conv=5), None),
                           (A, pf.chunk_mixer(heads=6, kv_heads=3, dim=12, vdim=18, size=31, scale=0.37, softcap=7.5), pf.dense(52, 1.75)),
                           (L, pf.latent_mixer(heads=5, dim=12, rot_dim=6, vdim=9, q_rank=26, kv_rank=22, scale=0.21, base=777.0, scaling=(2.5, 96, 8.0, 2.0)),
                            pf.dense(36, 2.25)),
                           (A, pf.chunk_mixer(heads=2, kv_heads=1, v_mix=False, size=0), None),
                           (A, pf.chunk_mixer(heads=9, kv_heads=3, dim=8, vdim=18, size=7), None)],
                          width=56, vocab=77, eps=3e-5, scale=2.5, mult=0.35, logit_softcap=17.0)


def test_spec_carries_every_size_and_constant():
    spec = config_from_dict(sample_config()).model_spec()
    assert (spec.hidden_size, spec.vocab_size) == (56, 77)
    assert [(e.layer, e.cache, e.writes, e.reenter) for e in spec.schedule] == [(i, i, True, False) for i in range(5)]
    assert [l.block for l in spec.layers] == ["sandwich_mixer", "sandwich", "sandwich", "sandwich_mixer", "sandwich_mixer"]
    for l in spec.layers:
        assert sorted(l.norms) == (["norm1", "norm1b", "norm2", "norm2b"] if l.block == "sandwich" else ["norm1", "norm1b"])
        for role, n in l.norms.items():
            assert n.kind == "rmsnorm" and n["eps"] == 3e-5 and n["size"] == 56 and n["post_scale"] == (0.35 if role.endswith("b") else 1.0)
    s, a, b, plain, third = (l.mixer for l in spec.layers)
    assert s.kind == "head_delta" and (s["n_heads"], s["n_kv_heads"], s["head_dim"], s["v_head_dim"], s["conv"], s["norm_eps"]) == (6, 3, 10, 14, 5, 3e-5)
    assert math.isclose(s["q_scale"], 10 ** -0.5)
    assert a.kind == "attention" and (a["n_heads"], a["n_kv_heads"], a["head_dim"], a["v_head_dim"], a["chunk"], a["scale"], a["softcap"]) == \
        (6, 3, 12, 18, 31, 0.37, 7.5)
    assert a["unit_sink"] is True and a["out_gate"] == "sigmoid" and a["position"].kind == "none"
    # values are kept by the first layer that mixes, mixed in the later ones, and left alone where v_mix is false
    assert a["value_mix"] == "first" and "value_mix" not in plain.params and third["value_mix"] == "mix"
    assert plain["chunk"] == 0 and third["chunk"] == 7
    assert b.kind == "latent_attention" and (b["n_heads"], b["head_dim"], b["rot_head_dim"], b["v_head_dim"], b["q_rank"], b["kv_rank"], b["scale"]) == \
        (5, 12, 6, 9, 26, 22, 0.21)
    pos = b["position"]
    assert pos.kind == "rope_half" and (pos["theta"], pos["rot_dim"], pos["head_dim"]) == (777.0, 6, 6)
    assert pos["scaling"] == {"factor": 2.5, "original": 96.0, "fast": 8.0, "slow": 2.0}
    assert b["out_gate"] == "head_sigmoid"
    f = spec.layers[1].ffn
    assert f.kind == "gated_mlp" and (f["intermediate_size"], f["activation"], f["activation_limit"]) == (52, "swish_clamped", 1.75)
    assert spec.layers[2].ffn["activation_limit"] == 2.25 and spec.layers[0].ffn.kind == ""
    assert spec.embedding["scale"] == 2.5 and spec.head["tied"] is True and spec.head["softcap"] == 17.0


def test_the_python_face_is_typed_and_round_trips():
    c = config_from_dict(sample_config())
    assert isinstance(c, FifotarConfig) and c.architecture == "Fifotar"
    assert FifotarConfig.from_dict(c.to_dict()) == c and c.to_dict()["width"] == 56


def test_declared_tensors_are_the_files_names_and_shapes():
    cfg = sample_config()
    decls = {name: tuple(shape) for name, (shape, _) in tensor_decls(config_from_dict(cfg)).items()}
    assert decls == {k: tuple(v[0]) for k, v in pf.tensor_shapes(cfg).items()}


@pytest.mark.parametrize("edit, word", [
    (lambda c: c["layers"][0].__setitem__("type", "convolution"), "unknown type"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("kv_heads", 4), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("conv", 0), "conv"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("softcap", 0.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"]["mask"].__setitem__("size", 0), "mask.size"),
    (lambda c: c["layers"][4]["mixer"].__setitem__("vdim", 20), "value channels"),
    (lambda c: c["layers"][2]["mixer"].__setitem__("q_rank", 0), "q_rank"),
    (lambda c: c["layers"][2]["mixer"]["rot"].__setitem__("dims", 5), "rot.dims"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][1]["mlp"].__setitem__("kind", "moe"), "kind"),
    (lambda c: c["layers"][1]["mlp"].pop("limit"), "limit"),
    (lambda c: c["norm"].__setitem__("eps", 0.0), "eps"),
    (lambda c: c.__setitem__("layers", []), "layers"),
])
def test_what_cannot_be_built_is_refused_in_words(edit, word):
    cfg = sample_config()
    edit(cfg)
    with pytest.raises(ConfigError) as e:
        tensor_decls(config_from_dict(cfg))
    assert word in str(e.value)


# ---------------------------------------------------------------- the plain implementation against second formulations


def test_delta_rule_against_its_linear_map_form():
    """S_t = g (I - beta k k^T) S_(t-1) + beta k v^T in one matrix step, read by q afterwards."""
    rng = np.random.default_rng(0)
    n, d, dv = 9, 5, 4
    q, k = rng.standard_normal((2, n, 1, d))
    k = pf.unit(k)
    v = rng.standard_normal((n, 2, dv))
    g, beta = rng.uniform(0.3, 1.0, (n, 2)), rng.uniform(0.1, 1.0, (n, 2))
    got = pf.delta_scan(q, k, v, g, beta, 2)
    for a in range(2):
        S = np.zeros((d, dv))
        for t in range(n):
            kt = k[t, 0][:, None]
            S = g[t, a] * (np.eye(d) - beta[t, a] * kt @ kt.T) @ S + beta[t, a] * kt @ v[t, a][None]
            assert np.allclose(got[t, a], S.T @ q[t, 0], rtol=1e-10, atol=1e-12)


def test_convolution_against_numpy():
    rng = np.random.default_rng(1)
    x, taps = rng.standard_normal((11, 3)), rng.standard_normal((3, 4))
    y = pf.causal_conv(x, taps)
    for c in range(3):
        assert np.allclose(y[:, c], np.convolve(x[:, c], taps[c, ::-1])[:11])


def test_head_decay_lies_between_zero_and_one():
    g = pf.head_decay(np.array([-30.0, 0.0, 30.0]), np.array([0.0, 0.0, 0.0]), np.zeros(3))
    assert np.allclose(g, [1.0, 0.5, math.exp(-30.0)])


def test_chunked_attention_against_its_matrix_form():
    rng = np.random.default_rng(2)
    m = pf.chunk_mixer(heads=4, kv_heads=2, dim=6, vdim=10, size=5, scale=0.7, softcap=2.0)
    cfg = pf.make_config([(A, m, None)])
    w = f64(pf.random_weights(cfg, 3, 1.5))
    n = 17
    h, first = rng.standard_normal((n, cfg["width"])), rng.standard_normal((n, 20))
    lam = float(w["l0.mix.vmix"])
    q = (h @ w["l0.mix.q"].T).reshape(n, 4, 6)
    k = np.repeat((h @ w["l0.mix.k"].T).reshape(n, 2, 6), 2, axis=1)
    own = h @ w["l0.mix.v"].T
    v = np.repeat((own + lam * (first - own)).reshape(n, 2, 10), 2, axis=1)
    s = 2.0 * np.tanh(np.einsum("ihd,jhd->hij", q, k) * 0.7 / 2.0)
    i, j = np.indices((n, n))
    s = np.where((j <= i) & (i // 5 == j // 5), s, -np.inf)
    p = np.exp(s) / (1.0 + np.exp(s).sum(-1, keepdims=True))
    o = np.einsum("hij,jhe->ihe", p, v).reshape(n, -1) / (1.0 + np.exp(-(h @ w["l0.mix.g"].T)))
    y, kept = pf.chunked_attention(h, w, "l0.mix.", m, first)
    assert np.allclose(y, o @ w["l0.mix.o"].T, rtol=1e-9, atol=1e-11) and np.array_equal(kept, own)
    assert not np.allclose(pf.chunked_attention(h, w, "l0.mix.", m, None)[0], y)


def test_half_rotation_against_complex_numbers():
    rng = np.random.default_rng(3)
    x = rng.standard_normal((3, 12))
    rot = {"base": 50.0, "dims": 8, "scaling": {"factor": 4.0, "original": 100, "fast": 6.0, "slow": 1.0}}
    # by hand: dim(t) = 8 ln(100 / (2 pi t)) / (2 ln 50); the ramp runs from 0 to 3
    dim = [8 * math.log(100 / (2 * math.pi * t)) / (2 * math.log(50.0)) for t in (6.0, 1.0)]
    assert math.floor(dim[0]) == 0 and math.ceil(dim[1]) == 3
    f = [50.0 ** (-i / 4) * ((1 - r) + r / 4) for i, r in enumerate([0.0, 1 / 3, 2 / 3, 1.0])]
    got, mag = pf.yarn_frequencies(rot)
    assert np.allclose(got, f) and math.isclose(mag, 0.1 * math.log(4.0) + 1.0)
    for p in (0, 1, 37):
        z = (x[:, :4] + 1j * x[:, 4:8]) * np.array([mag * cmath.exp(1j * p * fi) for fi in f])
        y = pf.rotate_halves(x, p, rot)
        assert np.allclose(y[:, :4], z.real) and np.allclose(y[:, 4:8], z.imag) and np.array_equal(y[:, 8:], x[:, 8:])


def test_latent_attention_against_its_absorbed_form():
    rng = np.random.default_rng(4)
    m = pf.latent_mixer(heads=3, dim=8, rot_dim=4, vdim=6, q_rank=10, kv_rank=14, scale=0.4, base=20.0)
    cfg = pf.make_config([(L, m, None)])
    w = f64(pf.random_weights(cfg, 5))
    n = 13
    h = rng.standard_normal((n, cfg["width"]))
    c0 = h @ w["l0.mix.dq"].T
    q = ((c0 / np.sqrt((c0 ** 2).mean(-1, keepdims=True) + 1e-5) * w["l0.mix.dq.norm"]) @ w["l0.mix.uq"].T).reshape(n, 3, 12)
    down = h @ w["l0.mix.dkv"].T
    c = down[:, :14] / np.sqrt((down[:, :14] ** 2).mean(-1, keepdims=True) + 1e-5) * w["l0.mix.dkv.norm"]
    uk, uv = w["l0.mix.uk"].reshape(3, 8, 14), w["l0.mix.uv"].reshape(3, 6, 14)
    gate = 1 / (1 + np.exp(-(h @ w["l0.mix.g"].T)))
    freqs, mag = pf.yarn_frequencies(m["rot"])
    out = np.zeros((n, 3, 6))
    for i in range(n):
        for a in range(3):
            qa = uk[a].T @ q[i, a, :8]
            zq, sc = q[i, a, 8:10] + 1j * q[i, a, 10:], []
            for j in range(i + 1):      # the rotated product depends on the distance, and carries the magnitude twice
                zk = down[j, 14:16] + 1j * down[j, 16:]
                turn = np.array([cmath.exp(1j * (j - i) * f) for f in freqs])
                sc.append((qa @ c[j] + mag * mag * (np.conj(zq) * zk * turn).real.sum()) * 0.4)
            p = np.exp(np.array(sc) - max(sc))
            p /= p.sum()
            out[i, a] = uv[a] @ (p @ c[:i + 1]) * gate[i, a]
    assert np.allclose(pf.latent_attention(h, w, "l0.mix.", m, 1e-5), out.reshape(n, -1) @ w["l0.mix.o"].T, rtol=1e-9, atol=1e-11)


def test_feed_forward_limits():
    """The gate is cut from above only, the up projection on both sides."""
    W = {"f.gate": np.array([[1.0]]), "f.up": np.array([[1.0]]), "f.down": np.array([[1.0]])}
    def f(x): return float(pf.clamped_mlp(np.array([[x]]), W, "f.", 2.0)[0, 0])
    assert math.isclose(f(5.0), 2.0 / (1 + math.exp(-1.702 * 2.0)) * 3.0)
    assert math.isclose(f(-5.0), -5.0 / (1 + math.exp(1.702 * 5.0)) * (-2.0 + 1.0))
    assert math.isclose(f(0.5), 0.5 / (1 + math.exp(-1.702 * 0.5)) * 1.5)


def test_zero_sink_and_soft_cap():
    s = np.array([-800.0, -801.0])
    assert np.allclose(pf.row_softmax_with_zero_sink(s), 0.0)            # everything goes to the sink
    assert np.allclose(pf.row_softmax_with_zero_sink(np.array([900.0, 900.0])), 0.5)
    assert math.isclose(float(pf.soft_cap(1e9, 3.0)), 3.0) and math.isclose(float(pf.soft_cap(1e-6, 3.0)), 1e-6, rel_tol=1e-9)


def test_values_are_mixed_with_the_first_mixing_layer_only():
    mix = dict(heads=2, kv_heads=1, dim=8, vdim=12)
    cfg = pf.make_config([(A, pf.chunk_mixer(**mix, v_mix=False), None), (A, pf.chunk_mixer(**mix), None), (A, pf.chunk_mixer(**mix), None)])
    w = f64(pf.random_weights(cfg, 1))
    ids = [3, 9, 27, 81, 5]
    ref = pf.forward(cfg, w, ids)
    for name, changes in (("l1.mix.vmix", False), ("l2.mix.vmix", True)):
        other = dict(w)
        other[name] = w[name] + 0.3
        assert np.array_equal(pf.forward(cfg, other, ids), ref) != changes
