"""The Fifotar decoder in the engine against the plain implementation (tests/plain_fifotar.py), GPU.

Every test makes its own small configuration and its own weights (numpy, rounded to bfloat16 so that the float32
mode, the bfloat16 mode and the plain implementation see the same numbers).  Weights are drawn so that faults show, and
where one key, one early token or the sink has to decide they are edited so that it does.
"""
import json
import os
import subprocess

import numpy as np
import pytest
import plain_fifotar as pf
from util import BF16_TOL, assert_close, rel_err

from inferllm_b200 import Engine, EngineOptions, Model, ModelConfig, StepItem

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
S, A, L = "delta", "attention", "latent_attention"
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def f64(w):
    return {k: np.asarray(v, np.float64) for k, v in w.items()}


def write_model(folder, cfg, seed, edit=None, gain=0.7):
    w = pf.random_weights(cfg, seed, gain)
    if edit:
        edit(w)
        w = {k: pf.bf16_round(np.asarray(v, np.float32)) for k, v in w.items()}
    pf.write_model(folder, cfg, w)
    return f64(w)


def engine(folder, dtype, max_tokens=2048, page_size=64, max_seq_len=1024, poison=False, max_batch=None):
    return Engine.from_folder(folder, EngineOptions(dtype=dtype, max_tokens=max_tokens, page_size=page_size, max_seq_len=max_seq_len,
                                                    poison_freed_pages=poison, max_batch=max_batch))


def whole(eng, ids):
    s = eng.new_sequence()
    lg = eng.step([StepItem(s, list(ids), list(range(len(ids))))]).cpu().numpy()
    eng.end_sequence(s)
    return lg


def in_portions(eng, ids, sizes):
    """The sequence in steps of the given sizes (the last size repeats)."""
    s, at, out, k = eng.new_sequence(), 0, [], 0
    while at < len(ids):
        n = min(sizes[min(k, len(sizes) - 1)], len(ids) - at)
        out.append(eng.step([StepItem(s, list(ids[at:at + n]), list(range(n)))]).cpu().numpy())
        at += n
        k += 1
    eng.end_sequence(s)
    return np.concatenate(out)


def same_or_close(a, b, dtype, what):
    """float32: every kernel fixes the order of its sums per row, so two ways of cutting the same tokens give the
    same bits; bfloat16: the library's products choose kernels by shape."""
    if dtype == "float32":
        assert np.array_equal(a, b), f"{what}: float32 logits differ between two cuttings (max {np.abs(a - b).max():.3e})"
    else:
        assert_close(a, b, dtype, what)


def prompt(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


CONFIGS = {
    # all three mixers, layers with and without a feed-forward, chunks shorter than a page, values mixed twice
    "mixed": pf.make_config([(S, pf.delta_mixer(), None), (A, pf.chunk_mixer(), pf.dense()), (S, pf.delta_mixer(), None),
                             (L, pf.latent_mixer(), pf.dense()), (A, pf.chunk_mixer(), pf.dense(24, 0.8)), (A, pf.chunk_mixer(), None)]),
    # another order, one key head per query head, no convolution, equal sizes, a layer that mixes no values between two
    # that do, chunks of different sizes, no rotation scaling, factors of 1
    "other": pf.make_config([(L, pf.latent_mixer(heads=2, dim=12, rot_dim=4, vdim=12, q_rank=12, kv_rank=20, scale=0.4, base=50.0, scaling=None), None),
                             (A, pf.chunk_mixer(heads=2, kv_heads=2, dim=16, vdim=16, size=33, softcap=3.0), pf.dense(28, 3.0)),
                             (A, pf.chunk_mixer(heads=4, kv_heads=1, dim=8, vdim=24, size=5, v_mix=False), None),
                             (S, pf.delta_mixer(heads=2, kv_heads=2, dim=16, vdim=16, conv=1), pf.dense(20)),
                             (A, pf.chunk_mixer(heads=6, kv_heads=2, dim=8, vdim=16, size=70), None)],
                            width=40, vocab=61, eps=1e-6, scale=1.0, mult=1.0, logit_softcap=50.0),
    # heads of 128 and 64 channels and a cache row of 128 (the tensor-core attention kernels), chunks across pages
    "wide": pf.make_config([(A, pf.chunk_mixer(heads=4, kv_heads=2, dim=128, vdim=128, size=150, scale=0.09, softcap=6.0), pf.dense(96)),
                            (S, pf.delta_mixer(heads=4, kv_heads=2, dim=64, vdim=32, conv=3), None),
                            (L, pf.latent_mixer(heads=4, dim=32, rot_dim=32, vdim=32, q_rank=48, kv_rank=96, scale=0.15), pf.dense(64)),
                            (A, pf.chunk_mixer(heads=6, kv_heads=3, dim=64, vdim=64, size=64, scale=0.12, softcap=4.0, v_mix=False), None)],
                           width=64, vocab=128),
    # an odd width and vocabulary, odd head sizes, more taps than the fast path of the convolution has
    "odd": pf.make_config([(S, pf.delta_mixer(heads=3, kv_heads=1, dim=7, vdim=11, conv=6), pf.dense(21)),
                           (A, pf.chunk_mixer(heads=3, kv_heads=1, dim=10, vdim=14, size=13), None),
                           (L, pf.latent_mixer(heads=3, dim=10, rot_dim=6, vdim=14, q_rank=15, kv_rank=27, scale=0.3), None)], width=45, vocab=71),
}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for i, (name, cfg) in enumerate(CONFIGS.items()):
        d = str(tmp_path_factory.mktemp("ff_" + name))
        out[name] = (d, cfg, write_model(d, cfg, 7 + i))
    return out


# ------------------------------------------------------------------ each mechanism alone

ALONE = {
    "delta": pf.make_config([(S, pf.delta_mixer(), None)]),
    "delta_one_head": pf.make_config([(S, pf.delta_mixer(heads=1, kv_heads=1, dim=24, vdim=8, conv=2), None)]),
    "delta_head_per_kv_head": pf.make_config([(S, pf.delta_mixer(heads=3, kv_heads=3, dim=16, vdim=40, conv=3), None)]),
    "delta_no_convolution": pf.make_config([(S, pf.delta_mixer(conv=1), None)]),
    "delta_many_taps": pf.make_config([(S, pf.delta_mixer(conv=9), None)]),
    "delta_many_heads": pf.make_config([(S, pf.delta_mixer(heads=24, kv_heads=3, dim=8, vdim=8), None)]),
    "delta_wide": pf.make_config([(S, pf.delta_mixer(heads=2, kv_heads=1, dim=130, vdim=70), None)], width=64),
    "delta_very_wide": pf.make_config([(S, pf.delta_mixer(heads=2, kv_heads=1, dim=260, vdim=36), None)], width=64),
    "chunks": pf.make_config([(A, pf.chunk_mixer(v_mix=False), None)]),
    "chunks_first_mixing_layer": pf.make_config([(A, pf.chunk_mixer(), None)]),
    "chunks_of_one": pf.make_config([(A, pf.chunk_mixer(size=1), None)]),
    "chunks_of_two": pf.make_config([(A, pf.chunk_mixer(size=2), None)]),
    "chunks_of_a_page": pf.make_config([(A, pf.chunk_mixer(size=64), None)]),
    "chunks_longer_than_the_sequence": pf.make_config([(A, pf.chunk_mixer(size=4000), None)]),
    "no_chunks": pf.make_config([(A, pf.chunk_mixer(size=0), None)]),
    "one_kv_head": pf.make_config([(A, pf.chunk_mixer(heads=6, kv_heads=1, dim=16, vdim=40), None)]),
    "head_per_kv_head": pf.make_config([(A, pf.chunk_mixer(heads=3, kv_heads=3, dim=40, vdim=8), None)]),
    "equal_sizes": pf.make_config([(A, pf.chunk_mixer(heads=4, kv_heads=2, dim=32, vdim=32), None)]),
    "low_cap": pf.make_config([(A, pf.chunk_mixer(scale=1.2, softcap=0.8), None)]),
    "heads_of_64": pf.make_config([(A, pf.chunk_mixer(heads=4, kv_heads=1, dim=64, vdim=64, size=50, scale=0.2, softcap=3.0), None)], width=64),
    "heads_of_128": pf.make_config([(A, pf.chunk_mixer(heads=2, kv_heads=2, dim=128, vdim=128, size=37, scale=0.1, softcap=3.0), None)], width=64),
    "keys_wider_than_values": pf.make_config([(A, pf.chunk_mixer(heads=4, kv_heads=2, dim=200, vdim=24, scale=0.07), None)], width=64),
    "values_wider_than_keys": pf.make_config([(A, pf.chunk_mixer(heads=4, kv_heads=4, dim=8, vdim=256, scale=0.4), None)], width=64),
    "odd_heads": pf.make_config([(A, pf.chunk_mixer(heads=2, kv_heads=1, dim=9, vdim=13), None)]),
    "mixed_values": pf.make_config([(A, pf.chunk_mixer(), None), (A, pf.chunk_mixer(), None), (A, pf.chunk_mixer(v_mix=False), None),
                                    (A, pf.chunk_mixer(heads=8, kv_heads=2, size=9), None)]),
    "latent": pf.make_config([(L, pf.latent_mixer(), None)]),
    "latent_unscaled_rotation": pf.make_config([(L, pf.latent_mixer(scaling=None), None)]),
    "latent_ramp_over_all_pairs": pf.make_config([(L, pf.latent_mixer(rot_dim=16, base=30.0, scaling=(8.0, 600, 50.0, 0.2)), None)]),
    "latent_step_ramp": pf.make_config([(L, pf.latent_mixer(rot_dim=12, base=1e4, scaling=(2.0, 40, 3.0, 3.0)), None)]),
    "latent_one_head_one_pair": pf.make_config([(L, pf.latent_mixer(heads=1, dim=24, rot_dim=2, vdim=8, q_rank=9, kv_rank=30), None)]),
    "latent_row_of_64_many_heads": pf.make_config([(L, pf.latent_mixer(heads=18, dim=8, rot_dim=16, vdim=8, kv_rank=48, scale=0.3), None)]),
    "latent_row_of_128": pf.make_config([(L, pf.latent_mixer(heads=5, dim=16, rot_dim=32, vdim=16, kv_rank=96, scale=0.2), None)]),
    "latent_row_of_136": pf.make_config([(L, pf.latent_mixer(heads=7, dim=20, rot_dim=24, vdim=16, kv_rank=112, scale=0.15), None)]),
    "latent_row_of_256": pf.make_config([(L, pf.latent_mixer(heads=9, dim=16, rot_dim=64, vdim=12, kv_rank=192, scale=0.15), None)]),
    "latent_row_of_576": pf.make_config([(L, pf.latent_mixer(heads=2, dim=32, rot_dim=64, vdim=32, q_rank=40, kv_rank=512, scale=0.06), None)], width=64),
    "latent_odd_row": pf.make_config([(L, pf.latent_mixer(heads=2, dim=12, rot_dim=6, vdim=10, q_rank=11, kv_rank=21), None)]),
    "feed_forward": pf.make_config([(S, pf.delta_mixer(), pf.dense(72, 0.9))]),
    "feed_forward_wide_limit": pf.make_config([(A, pf.chunk_mixer(), pf.dense(30, 40.0))]),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ALONE))
def test_mechanism_alone(tmp_path, name, dtype):
    cfg = ALONE[name]
    w = write_model(str(tmp_path), cfg, 3)
    ids = prompt(cfg, 141, 5)
    ref = pf.forward(cfg, w, ids)
    eng = engine(str(tmp_path), dtype)
    got = whole(eng, ids)
    assert_close(got, ref, dtype, name)
    # and token by token through the cache
    one = in_portions(eng, ids, [1])
    assert_close(one, ref, dtype, name + " token by token")
    same_or_close(one, got, dtype, name + " token by token")


@pytest.mark.parametrize("dtype", DTYPES)
def test_constants_are_read(tmp_path, dtype):
    """The embedding's scale, the factor on the sublayers, the cap on the logits and eps, each far from the usual."""
    base = dict(width=48, scale=0.05, mult=2.5, logit_softcap=12.0, eps=0.02)
    cfg = pf.make_config([(A, pf.chunk_mixer(), pf.dense()), (S, pf.delta_mixer(), None), (L, pf.latent_mixer(), None)], **base)
    w = write_model(str(tmp_path), cfg, 4)
    ids = prompt(cfg, 60, 2)
    ref = pf.forward(cfg, w, ids)
    for key, other in (("scale", 0.06), ("mult", 2.0), ("logit_softcap", 13.0), ("eps", 1e-5)):
        alt = pf.make_config([(x["type"], x["mixer"], x["mlp"]) for x in cfg["layers"]], **dict(base, **{key: other}))
        assert rel_err(pf.forward(alt, w, ids), ref) > 1e-3, key
    eng = engine(str(tmp_path), dtype)
    assert_close(whole(eng, ids), ref, dtype, "prompt")
    assert_close(in_portions(eng, ids, [50, 1]), ref, dtype, "decoding")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompt_through_the_tile_kernels(tmp_path, dtype):
    """A prompt long enough for the prompt kernels' tiles of queries and keys, on heads of 128, of unequal sizes and on
    latent rows of 128 and of 96, with the feed-forward's product on pairs of SMs."""
    cfg = pf.make_config([(A, pf.chunk_mixer(heads=4, kv_heads=2, dim=128, vdim=128, size=260, scale=0.09, softcap=5.0), pf.dense(256)),
                          (L, pf.latent_mixer(heads=4, dim=32, rot_dim=32, vdim=32, q_rank=64, kv_rank=96, scale=0.15), None),
                          (A, pf.chunk_mixer(heads=4, kv_heads=2, dim=48, vdim=72, size=333, scale=0.15, softcap=5.0, v_mix=False), None),
                          (L, pf.latent_mixer(heads=4, dim=32, rot_dim=16, vdim=32, q_rank=64, kv_rank=80, scale=0.15), None),
                          (S, pf.delta_mixer(heads=4, kv_heads=2, dim=64, vdim=64), None)], width=64)
    w = write_model(str(tmp_path), cfg, 21)
    ids = prompt(cfg, 600, 8)
    ref = pf.forward(cfg, w, ids)
    eng = engine(str(tmp_path), dtype, max_tokens=2048)
    got = whole(eng, ids)
    assert_close(got, ref, dtype, "600 tokens in one step")
    same_or_close(in_portions(eng, ids, [510, 1]), got, dtype, "the same, its last tokens one by one")
    same_or_close(in_portions(eng, ids, [250, 200, 150]), got, dtype, "three long portions")


GROUPS = {
    # query heads per key/value head that fill the single-token kernel's groups of heads exactly, partly and several times over
    "group_of_8": pf.make_config([(A, pf.chunk_mixer(heads=8, kv_heads=1, dim=16, vdim=32, size=50), None)], width=64),
    "group_of_3": pf.make_config([(A, pf.chunk_mixer(heads=6, kv_heads=2, dim=8, vdim=16, size=40), None)]),
    "group_of_7": pf.make_config([(A, pf.chunk_mixer(heads=7, kv_heads=1, dim=24, vdim=8, size=33), None)], width=56),
    "group_of_20": pf.make_config([(A, pf.chunk_mixer(heads=40, kv_heads=2, dim=8, vdim=24, size=77), None)], width=64),
    "40_heads_of_128": pf.make_config([(A, pf.chunk_mixer(heads=40, kv_heads=1, dim=128, vdim=128, size=77, scale=0.1), None)], width=64),
    "latent_40_heads_row_of_128": pf.make_config([(L, pf.latent_mixer(heads=40, dim=8, rot_dim=16, vdim=8, kv_rank=112, scale=0.2), None)], width=64),
    "wider": pf.make_config([(A, pf.chunk_mixer(heads=8, kv_heads=4, dim=32, vdim=16), pf.dense(300)), (S, pf.delta_mixer(heads=8, kv_heads=4, dim=32, vdim=32), None),
                             (L, pf.latent_mixer(heads=8, dim=24, rot_dim=16, vdim=24, q_rank=96, kv_rank=48), pf.dense(200))], width=192, vocab=301),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(GROUPS))
def test_other_sizes(tmp_path, name, dtype):
    cfg = GROUPS[name]
    w = write_model(str(tmp_path), cfg, 13)
    ids = prompt(cfg, 90, 7)
    ref = pf.forward(cfg, w, ids)
    eng = engine(str(tmp_path), dtype)
    assert_close(whole(eng, ids), ref, dtype, name)
    assert_close(in_portions(eng, ids, [70, 1]), ref, dtype, name + ", its last tokens one by one")
    a, b = ids[:55], ids[20:90]
    sa, sb = eng.new_sequence(), eng.new_sequence()
    eng.step([StepItem(sa, a[:40], []), StepItem(sb, b[:66], [])])
    got = [eng.step([StepItem(sa, [a[40 + i]], [0]), StepItem(sb, [b[66 + i]], [0])]).cpu().numpy() for i in range(4)]
    eng.end_sequence(sa)
    eng.end_sequence(sb)
    assert_close(np.stack([g[0] for g in got]), pf.forward(cfg, w, a)[40:44], dtype, name + ", two sequences decoded together, the first")
    assert_close(np.stack([g[1] for g in got]), pf.forward(cfg, w, b)[66:70], dtype, name + ", two sequences decoded together, the second")


# ------------------------------------------------------------------ whole models


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_first_tokens_and_one_token(models, name, dtype):
    d, cfg, w = models[name]
    eng = engine(d, dtype)
    for n in (1, 2, 3):
        ids = prompt(cfg, n, 20 + n)
        assert_close(whole(eng, ids), pf.forward(cfg, w, ids), dtype, f"{name} {n} tokens")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_portions_and_decoding(models, name, dtype):
    """Prefill against token-by-token decoding and portions of several sizes, down to two tokens, across page borders
    and chunk edges."""
    d, cfg, w = models[name]
    ids = prompt(cfg, 200, 13)
    layers = []
    ref = pf.forward(cfg, w, ids, layers)
    assert len(layers) == len(cfg["layers"])
    eng = engine(d, dtype)
    base = whole(eng, ids)
    assert_close(base, ref, dtype, name)
    for sizes in ([1], [2], [63, 2, 64, 7], [128, 1], [5, 64, 3], [1, 1, 2, 3, 50]):
        got = in_portions(eng, ids, sizes)
        assert_close(got, ref, dtype, f"{name} portions {sizes}")
        same_or_close(got, base, dtype, f"{name} portions {sizes}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_unequal_batches(models, name, dtype):
    """Requests of different lengths in one batch, then decoded together while the shorter ones end, against each alone."""
    d, cfg, w = models[name]
    eng = engine(d, dtype, max_tokens=4096)
    lens, extra = [1, 37, 150, 66], [9, 30, 12, 5]
    seqs = [prompt(cfg, n + e, 40 + i) for i, (n, e) in enumerate(zip(lens, extra))]
    refs = [pf.forward(cfg, w, s) for s in seqs]
    alone = [whole(eng, s) for s in seqs]
    slots = [eng.new_sequence() for _ in seqs]
    lg = eng.step([StepItem(slots[i], seqs[i][:lens[i]], list(range(lens[i]))) for i in range(len(seqs))]).cpu().numpy()
    at, got = 0, []
    for i, n in enumerate(lens):
        got.append([lg[at:at + n]])
        at += n
    pos = list(lens)
    live = list(range(len(seqs)))
    while live:
        lg = eng.step([StepItem(slots[i], [seqs[i][pos[i]]], [0]) for i in live]).cpu().numpy()
        for r, i in enumerate(live):
            got[i].append(lg[r:r + 1])
            pos[i] += 1
        for i in list(live):
            if pos[i] == len(seqs[i]):
                eng.end_sequence(slots[i])
                live.remove(i)
    for i in range(len(seqs)):
        g = np.concatenate(got[i])
        assert_close(g, refs[i], dtype, f"{name} batch, sequence {i}")
        same_or_close(g, alone[i], dtype, f"{name} batch, sequence {i} against itself alone")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_slots_and_pages_used_again(models, name, dtype):
    """A small cache whose slots and pages go round several times, freed pages poisoned with NaN: a sequence must never
    read a page that it does not hold, state starts at zero in a slot used before, and pages of finished chunks are
    given back while their sequence goes on."""
    d, cfg, w = models[name]
    eng = engine(d, dtype, max_tokens=320, max_batch=3, max_seq_len=256, poison=True)
    for rnd in range(4):
        seqs = [prompt(cfg, n, 70 + 10 * rnd + i) for i, n in enumerate((90 + rnd, 33, 70))]
        slots = [eng.new_sequence() for _ in seqs]
        cut = [len(s) // 2 + rnd for s in seqs]
        eng.step([StepItem(slots[i], seqs[i][:cut[i]], []) for i in range(3)])
        eng.end_sequence(slots[1])                        # its slot and pages go to the next sequence at once
        late = prompt(cfg, 40, 90 + rnd)
        s_late = eng.new_sequence()
        got_late = eng.step([StepItem(s_late, late, list(range(40)))]).cpu().numpy()
        assert_close(got_late, pf.forward(cfg, w, late), dtype, f"round {rnd}: a sequence in a slot used before")
        for i in (0, 2):
            rest = seqs[i][cut[i]:]
            got = eng.step([StepItem(slots[i], rest, list(range(len(rest))))]).cpu().numpy()
            assert_close(got, pf.forward(cfg, w, seqs[i])[cut[i]:], dtype, f"round {rnd}: sequence {i} continued")
            eng.end_sequence(slots[i])
        eng.end_sequence(s_late)


# ------------------------------------------------------------------ crafted cases


def crafted_ids(cfg, n, seed, at):
    """Random tokens in which token 7 stands at position `at` and nowhere else."""
    ids = [t if t != 7 else 8 for t in prompt(cfg, n, seed)]
    ids[at] = 7
    return ids


def spike(w, value=6.0):
    """Token 7's embedding is a spike in channel 5, which no other token has; channel 6 is a constant of all tokens."""
    w["embed"][:, 5] = 0.0
    w["embed"][:, 6] = 2.0
    w["embed"][7] = 0.0
    w["embed"][7, 5] = value
    w["embed"][7, 6] = 2.0
    w["l0.norm1"][5] = w["l0.norm1"][6] = 1.0
    w["l0.norm1b"][:] = 3.0 * np.asarray(w["l0.norm1b"])          # the mixer's share of the logits


def with_chunk(cfg, size):
    c = json.loads(json.dumps(cfg))
    for layer in c["layers"]:
        if layer["type"] == A:
            layer["mixer"]["mask"] = {"size": size}
    return c


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk,page,dims", [(64, 64, (8, 16)), (65, 64, (8, 16)), (63, 64, (8, 12)), (7, 16, (8, 16)), (33, 16, (9, 11)), (2, 64, (8, 16)),
                                             (64, 64, (128, 128)), (65, 64, (128, 128)), (130, 64, (64, 64)), (100, 64, (64, 64)), (150, 64, (16, 64))])
@pytest.mark.parametrize("place", ["first", "last"])
def test_one_key_decides_at_a_chunks_edge(tmp_path, chunk, page, dims, place, dtype):
    """The key of one position is made to stand out for every query that sees it: its token appears once, its embedding is
    a spike in one channel which the keys read, and the queries carry a constant.  At a chunk's first position it decides
    the whole chunk, up to the last position, and nothing after; at a chunk's last position it decides that position alone.
    The plain implementation with a chunk one longer or shorter must disagree, or the test would show nothing."""
    m = pf.chunk_mixer(heads=2, kv_heads=1, dim=dims[0], vdim=dims[1], size=chunk, scale=1.0, softcap=30.0, v_mix=False)
    cfg = pf.make_config([(A, m, None)], vocab=50)
    start = max(2, -(-64 // chunk)) * chunk                       # a chunk's first position, not the sequence's
    at = start if place == "first" else start - 1
    ids = crafted_ids(cfg, start + chunk + 40, 3, at)

    def edit(w):
        spike(w)
        for head in range(2):
            w["l0.mix.q"][head * dims[0]:(head + 1) * dims[0]] *= 0.3
            w["l0.mix.q"][head * dims[0]] = 0.0
            w["l0.mix.q"][head * dims[0], 6] = 1.5
        w["l0.mix.k"][:] = 0.3 * np.asarray(w["l0.mix.k"])
        w["l0.mix.k"][0] = 0.0
        w["l0.mix.k"][0, 5] = 2.0

    w = write_model(str(tmp_path), cfg, 9, edit)
    ref = pf.forward(cfg, w, ids)
    lo, hi = max(0, start - 3), min(len(ids), start + chunk + 3)
    for other in (chunk - 1, chunk + 1):
        if other > 0:
            assert rel_err(pf.forward(with_chunk(cfg, other), w, ids)[lo:hi], ref[lo:hi]) > 0.05, "the crafted key does not decide"
    eng = engine(str(tmp_path), dtype, page_size=page)
    assert_close(whole(eng, ids), ref, dtype, f"chunk {chunk}, prompt")
    assert_close(in_portions(eng, ids, [at, 1]), ref, dtype, f"chunk {chunk}, decoding from the key on")
    assert_close(in_portions(eng, ids, [start, 2]), ref, dtype, f"chunk {chunk}, portions from the edge on")
    assert_close(in_portions(eng, ids, [start - 1, 1, chunk - 1, 1, 1, 40]), ref, dtype, f"chunk {chunk}, steps at the edges")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dims", [(8, 24), (64, 64), (128, 128)])
def test_the_sink_decides(tmp_path, dims, dtype):
    """Scores far below zero for all keys: nearly all weight goes to the sink, and the head's output is a small part of a
    value (the norm behind the sublayer blows it up again unless the sink differs from row to row)."""
    m = pf.chunk_mixer(heads=2, kv_heads=1, dim=dims[0], vdim=dims[1], size=50, scale=1.0, softcap=20.0, v_mix=False)
    cfg = pf.make_config([(A, m, None)], vocab=50, eps=1e-2)

    def edit(w):
        w["embed"][:, 6] = 2.0
        w["l0.norm1"][6] = 1.0
        for head in range(2):
            w["l0.mix.q"][head * dims[0]:(head + 1) * dims[0]] *= 0.1
            w["l0.mix.q"][head * dims[0], 6] = 1.2
        w["l0.mix.k"][:] = 0.1 * np.asarray(w["l0.mix.k"])
        w["l0.mix.k"][0, 6] = -0.6

    w = write_model(str(tmp_path), cfg, 9, edit)
    ids = prompt(cfg, 160, 3)
    ref = pf.forward(cfg, w, ids)
    zero_sink = pf.row_softmax_with_zero_sink
    try:
        pf.row_softmax_with_zero_sink = pf.row_softmax
        assert rel_err(pf.forward(cfg, w, ids), ref) > 0.05, "the sink does not decide"
    finally:
        pf.row_softmax_with_zero_sink = zero_sink
    eng = engine(str(tmp_path), dtype)
    assert_close(whole(eng, ids), ref, dtype, "prompt")
    assert_close(in_portions(eng, ids, [70, 1]), ref, dtype, "decoding")
    assert_close(in_portions(eng, ids, [2]), ref, dtype, "portions of two")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("page,rank", [(64, 24), (16, 24), (64, 120), (64, 21), (64, 152)])
def test_one_far_key_decides_through_the_shared_rotated_part(tmp_path, page, rank, dtype):
    """With a huge base all pairs but the first hardly turn, so a spike in the second pair of one position's rotated key
    part, against queries that carry a constant there, stands out whatever the distance: hundreds of positions back, at a
    page border, in a prompt and in decoding.  (rank 120: cache rows of 128 channels, the tensor-core kernels in bfloat16;
    152: rows of 160; 21: a row that is no multiple of 8.)"""
    m = pf.latent_mixer(heads=2, dim=8, rot_dim=8, vdim=12, q_rank=16, kv_rank=rank, scale=1.0, base=1e30, scaling=None)
    cfg = pf.make_config([(L, m, None)], vocab=50)
    far = 63
    ids = crafted_ids(cfg, 300, 3, far)

    def edit(w):
        spike(w)
        w["l0.mix.dq"][0] = 0.0                           # channel 0 of the query latent: the constant
        w["l0.mix.dq"][0, 6] = 3.0
        w["l0.mix.dq.norm"][0] = 1.0
        for head in range(2):
            w["l0.mix.uq"][head * 16 + 8:head * 16 + 16] = 0.0
            w["l0.mix.uq"][head * 16 + 9, 0] = 2.0        # channel 1 of the rotated part: the second pair
        w["l0.mix.dkv"][rank + 1] = 0.0
        w["l0.mix.dkv"][rank + 1, 5] = 2.0
        w["l0.mix.g"][:] = 0.3 * np.asarray(w["l0.mix.g"])

    w = write_model(str(tmp_path), cfg, 9, edit)
    ref = pf.forward(cfg, w, ids)
    alt = pf.forward(cfg, w, ids[:far] + [8] + ids[far + 1:])
    assert rel_err(alt[200:], ref[200:]) > 0.05, "the crafted key does not decide"
    eng = engine(str(tmp_path), dtype, page_size=page)
    assert_close(whole(eng, ids), ref, dtype, "prompt")
    assert_close(in_portions(eng, ids, [60, 1]), ref, dtype, "decoding past the key")
    assert_close(in_portions(eng, ids, [far + 1, 2]), ref, dtype, "portions from the key on")
    assert_close(in_portions(eng, ids, [far, 1, 130, 7]), ref, dtype, "the key alone in a step")


@pytest.mark.parametrize("dtype", DTYPES)
def test_rotation_sees_the_distance_only(tmp_path, dtype):
    """Sharp attention through the rotated parts alone: the latent's keys are switched off, so a score depends on the
    rotated pairs, whose product is a function of the distance (times the squared magnitude).  The plain implementation
    with another base or without the scaling must disagree."""
    m = pf.latent_mixer(heads=2, dim=8, rot_dim=16, vdim=12, q_rank=20, kv_rank=24, scale=1.0, base=30.0, scaling=(6.0, 90, 8.0, 1.0))
    cfg = pf.make_config([(L, m, None)])

    def edit(w):
        w["l0.mix.uk"][:] = 0.0

    w = write_model(str(tmp_path), cfg, 12, edit, gain=1.0)
    ids = prompt(cfg, 230, 4)
    ref = pf.forward(cfg, w, ids)
    for key, value in (("base", 31.0), ("scaling", None)):
        alt = json.loads(json.dumps(cfg))
        alt["layers"][0]["mixer"]["rot"][key] = value
        assert rel_err(pf.forward(alt, w, ids)[50:], ref[50:]) > 0.01
    eng = engine(str(tmp_path), dtype)
    assert_close(whole(eng, ids), ref, dtype, "prompt")
    assert_close(in_portions(eng, ids, [190, 1]), ref, dtype, "decoding")
    assert_close(in_portions(eng, ids, [39, 2, 41, 64, 3]), ref, dtype, "portions")


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_state_remembers_one_early_token(tmp_path, dtype):
    """Decays next to 1 and one token whose key no other token comes near: what it wrote stays in the state, and the
    queries read it hundreds of tokens later, across steps of every size."""
    m = pf.delta_mixer(heads=4, kv_heads=2, dim=8, vdim=12, conv=3)
    cfg = pf.make_config([(S, m, None)], vocab=50)
    ids = crafted_ids(cfg, 300, 3, 17)

    def edit(w):
        spike(w)
        w["l0.mix.A_log"][:] = -3.0
        w["l0.mix.dt_bias"][:] = -5.0
        for kv in range(2):
            k, q = w["l0.mix.k"], w["l0.mix.q"]
            k[:, 5] = 0.0
            k[kv * 8] = 0.0
            k[kv * 8, 5] = 4.0                            # channel 0: the spike alone
            q[kv * 8] = 0.0
            q[kv * 8, 6] = 4.0                            # and the queries' constant
        for t in ("q", "k"):
            w["l0.mix.%s.conv" % t][:] = 0.0
            w["l0.mix.%s.conv" % t][:, -1] = 1.0

    w = write_model(str(tmp_path), cfg, 9, edit)
    ref = pf.forward(cfg, w, ids)
    alt = pf.forward(cfg, w, ids[:17] + [8] + ids[18:])
    assert rel_err(alt[250:], ref[250:]) > 0.05, "the early token does not decide"
    eng = engine(str(tmp_path), dtype)
    assert_close(whole(eng, ids), ref, dtype, "prompt")
    assert_close(in_portions(eng, ids, [18, 1]), ref, dtype, "decoding")
    assert_close(in_portions(eng, ids, [17, 1, 100, 2]), ref, dtype, "the token alone in a step")


@pytest.mark.parametrize("dtype", DTYPES)
def test_convolution_reaches_back_its_taps_and_no_further(tmp_path, dtype):
    """The oldest tap dominates: a token decides the row taps - 1 tokens later, whether the step is cut between them or not."""
    m = pf.delta_mixer(heads=2, kv_heads=1, dim=8, vdim=12, conv=4)
    cfg = pf.make_config([(S, m, None)], vocab=50)

    def edit(w):
        for t in ("q", "k", "v"):
            w["l0.mix.%s.conv" % t][:, 0] = 2.0
            w["l0.mix.%s.conv" % t][:, 1:] *= 0.2

    w = write_model(str(tmp_path), cfg, 9, edit)
    ids = prompt(cfg, 40, 6)
    ref = pf.forward(cfg, w, ids)
    eng = engine(str(tmp_path), dtype)
    for sizes in ([40], [1], [2], [3], [4], [5, 1, 1, 7], [17, 3, 2]):
        assert_close(in_portions(eng, ids, sizes), ref, dtype, f"portions {sizes}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_feed_forward_at_its_limits(tmp_path, dtype):
    """Gate and up projections far beyond the limit on both sides (the gate is cut from above only)."""
    cfg = pf.make_config([(A, pf.chunk_mixer(), pf.dense(64, 0.75))])

    def edit(w):
        w["l0.mlp.gate"] = 5.0 * np.asarray(w["l0.mlp.gate"])
        w["l0.mlp.up"] = 5.0 * np.asarray(w["l0.mlp.up"])

    w = write_model(str(tmp_path), cfg, 31, edit)
    ids = prompt(cfg, 600, 6)
    ref = pf.forward(cfg, w, ids)
    wide = json.loads(json.dumps(cfg))
    wide["layers"][0]["mlp"]["limit"] = 50.0
    assert rel_err(pf.forward(wide, w, ids), ref) > 0.02
    eng = engine(str(tmp_path), dtype)
    assert_close(whole(eng, ids), ref, dtype, "prompt (the product on pairs of SMs)")
    assert_close(in_portions(eng, ids, [100, 30, 1, 1, 200]), ref, dtype, "portions and single tokens")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(models, dtype):
    """Three hundred tokens one by one behind a short prompt: past several pages and chunks."""
    d, cfg, w = models["mixed"]
    ids = prompt(cfg, 330, 17)
    assert_close(in_portions(engine(d, dtype), ids, [30, 1]), pf.forward(cfg, w, ids), dtype, "long decoding")


# ------------------------------------------------------------------ the library's own entry points


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_model_api(models, dtype):
    """Model.generate: the scheduler batches the requests, decodes them together and ends each by itself."""
    d, cfg, w = models["mixed"]
    prompts = [prompt(cfg, n, 50 + n) for n in (3, 17, 70, 1)]
    m = Model(ModelConfig(compt_type=dtype, nr_ctx=256, max_tokens=1024))
    m.load(d)
    m.init(top_k=0, top_p=1.0, temp=0.0, repeat_penalty=1.0, repeat_last_n=0, seed=0, end_token=-1)
    got = m.generate(prompts, max_new_tokens=12, stop_ids=[]).tokens
    if dtype == "float32":
        assert got == [pf.greedy_generate(cfg, w, p, 12) for p in prompts]
        return
    # bfloat16 may turn a near-tie: every token the engine chose must be (within rounding) the best continuation of what
    # it had generated so far, by the plain implementation's logits for that very sequence
    for p, g in zip(prompts, got):
        assert len(g) == 12
        lg = pf.forward(cfg, w, p + g)[len(p) - 1:-1]
        gap = lg.max(-1) - lg[np.arange(12), g]
        assert (gap <= BF16_TOL * np.abs(lg).max()).all(), (g, gap)


def test_command_line(models):
    """bin/llama on a Fifotar folder: greedy tokens of two requests, float32."""
    d, cfg, w = models["other"]
    prompts = [prompt(cfg, n, 90 + n) for n in (7, 12)]
    want = [pf.greedy_generate(cfg, w, p, 6) for p in prompts]
    args = [os.path.join(ROOT, "bin", "llama"), "-m", d, "-d", "float32", "-c", "128", "-n", "6", "--temp", "0", "--top_k", "0",
            "--top_p", "1", "--repeat_penalty", "1", "-s", "1"]
    for p in prompts:
        args += ["--prompt-ids", ",".join(map(str, p))]
    r = subprocess.run(args, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    got = [[int(t) for t in ln.split(": ")[1].split(",")] for ln in r.stdout.splitlines() if ln.startswith("[")]
    assert got == want


def test_trace_replay_program(models, tmp_path):
    d, cfg, w = models["mixed"]
    a, b = prompt(cfg, 40, 1), prompt(cfg, 9, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:33], "want": [0, 32]}, {"id": "b", "tokens": b[:8], "want": [7]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[33:34], "want": [0]}, {"id": "b", "tokens": b[8:], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[34:35], "want": [0]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[35:], "want": [4]}], "end": ["a"]}]
    out = str(tmp_path / "out")
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", out, "--max-tokens", "128"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done %d" % i for i in range(4)]
    ra, rb = pf.forward(cfg, w, a), pf.forward(cfg, w, b)
    V = cfg["vocab"]
    got0 = np.fromfile(os.path.join(out, "0.f32"), "<f4").reshape(-1, V)
    assert_close(got0, np.stack([ra[0], ra[32], rb[7]]), "float32", "step 0")
    assert_close(np.fromfile(os.path.join(out, "1.f32"), "<f4").reshape(-1, V), ra[33:34], "float32", "step 1")
    assert_close(np.fromfile(os.path.join(out, "2.f32"), "<f4").reshape(-1, V), ra[34:35], "float32", "step 2")
    assert_close(np.fromfile(os.path.join(out, "3.f32"), "<f4").reshape(-1, V), ra[39:40], "float32", "step 3")
