"""The Zeluzen decoder in the engine against the plain implementation (tests/plain_zeluzen.py), GPU.

Every test makes its own small configuration and its own weights (numpy, rounded to bfloat16 so that the float32
mode, the bfloat16 mode and the plain implementation see the same numbers).  Weights are drawn so that faults show, and
where one key, one early token, the sink or the bonus has to decide they are edited so that it does.
"""
import json
import os
import subprocess

import numpy as np
import pytest
import plain_zeluzen as pz
from util import BF16_TOL, assert_close, rel_err

from inferllm_b200 import Engine, EngineOptions, Model, ModelConfig, StepItem

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
S, A = "wkv", "attention"
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def f64(w):
    return {k: np.asarray(v, np.float64) for k, v in w.items()}


class Weights(dict):
    """The weights and the tokens that a prompt may have (None: all)."""
    tokens = None


def write_model(folder, cfg, seed, edit=None, gain=0.7, rank=7, dtype="float32"):
    """In bfloat16 the routers are made so that rounding cannot turn a choice (which changes a token's row by far more than
    rounding); in float32 they read the whole stream."""
    w = pz.random_weights(cfg, seed, gain, rank)
    if edit:
        edit(w)
        w = {k: pz.bf16_round(np.asarray(v, np.float32)) for k, v in w.items()}
    tokens = pz.steady_routing(cfg, w) if dtype == "bfloat16" and any((L.get("mlp") or {}).get("kind") == "moe" for L in cfg["layers"]) else None
    pz.write_model(folder, cfg, w)
    out = Weights(f64(w))
    out.tokens = tokens
    assert tokens is None or len(tokens) >= 8, len(tokens)
    return out


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


def close(got, ref, dtype, what):
    """float32: every position within the bound.  bfloat16: a head's unit norm enlarges what rounding leaves of a nearly empty
    output: at most one position in fifty (or one) may exceed the bound, none five times the bound, and the others are held
    to it."""
    got, ref = np.asarray(got, np.float64), np.asarray(ref, np.float64)
    if dtype == "float32":
        return assert_close(got, ref, dtype, what)
    assert np.isfinite(got).all(), f"{what}: non-finite values"
    err = np.abs(got - ref).max(-1) / max(np.abs(ref).max(), 1e-30)
    over = err > BF16_TOL
    assert over.sum() <= max(1, len(err) // 50), f"{what}: {int(over.sum())} of {len(err)} positions exceed {BF16_TOL:.1e} (worst {err.max():.3e})"
    assert err.max() <= 5 * BF16_TOL, f"{what}: a position is off by {err.max():.3e}"
    if (~over).any():
        assert_close(got[~over], ref[~over], dtype, what)


def same_or_close(a, b, dtype, what):
    """float32: every kernel fixes the order of its sums per row, so two ways of cutting the same tokens give the
    same bits; bfloat16: the library's products choose kernels by shape, and prompts take sixteen tokens' sums together."""
    if dtype == "float32":
        assert np.array_equal(a, b), f"{what}: float32 logits differ between two cuttings (max {np.abs(a - b).max():.3e})"
    else:
        close(a, b, dtype, what)


def prompt(cfg, n, seed, w=None):
    ids = np.random.default_rng(seed).integers(0, 1 << 30, n)
    tokens = getattr(w, "tokens", None)
    return (ids % cfg["vocab"]).tolist() if tokens is None else [tokens[i % len(tokens)] for i in ids]


MOE = pz.moe_mlp
CONFIGS = {
    # both mixers, all kinds of feed-forward and none, chunks shorter than a page, readers with masks of their own
    "mixed": pz.make_config([(S, pz.wkv_mixer(), pz.dense_mlp()), (A, pz.attn_mixer(), MOE()), (S, pz.wkv_mixer(heads=2, dim=24), None),
                             (A, pz.attn_mixer(heads=4, size=33, kv_from=1), MOE(ff=16, experts=3, identity=4, top=2)), (S, pz.wkv_mixer(), MOE()),
                             (A, pz.attn_mixer(heads=2, size=0, kv_from=1), None)]),
    # another order, equal sizes, one head, no scaling, no identity experts, every expert chosen
    "other": pz.make_config([(A, pz.attn_mixer(heads=2, kv_heads=2, dim=16, vdim=16, size=33, dims=16, scaling=None), MOE(ff=12, experts=4, identity=0, top=1)),
                             (S, pz.wkv_mixer(heads=1, dim=32), MOE(ff=20, experts=2, identity=1, top=3)), (S, pz.wkv_mixer(heads=5, dim=8), None),
                             (A, pz.attn_mixer(heads=4, kv_heads=1, dim=8, vdim=24, size=5, dims=4), pz.dense_mlp(28))], width=40, vocab=61, eps=1e-6),
    # heads of 128 and 64 channels (the tensor-core attention kernels), chunks across pages, wide recurrent heads
    "wide": pz.make_config([(A, pz.attn_mixer(heads=4, kv_heads=2, dim=128, vdim=128, size=150, scale=0.09, dims=64), pz.dense_mlp(96)),
                            (S, pz.wkv_mixer(heads=2, dim=128), MOE(ff=64, experts=6, identity=2, top=2)),
                            (A, pz.attn_mixer(heads=8, kv_heads=2, dim=128, vdim=128, size=64, scale=0.1, dims=64, kv_from=0), None),
                            (A, pz.attn_mixer(heads=6, kv_heads=3, dim=64, vdim=64, size=64, scale=0.12, dims=32), MOE(ff=32, experts=4, identity=1, top=2)),
                            (S, pz.wkv_mixer(heads=3, dim=64), None)], width=64, vocab=128),
    # an odd width and vocabulary, odd head sizes
    "odd": pz.make_config([(S, pz.wkv_mixer(heads=3, dim=7), pz.dense_mlp(21)), (A, pz.attn_mixer(heads=3, kv_heads=1, dim=10, vdim=14, size=13, dims=6), None),
                           (S, pz.wkv_mixer(heads=2, dim=11), MOE(ff=9, experts=3, identity=1, top=2))], width=45, vocab=71),
}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for i, (name, cfg) in enumerate(CONFIGS.items()):
        for dtype in DTYPES:
            d = str(tmp_path_factory.mktemp("zz_" + name + dtype))
            out[name, dtype] = (d, cfg, write_model(d, cfg, 7 + i, dtype=dtype))
    return out


# ------------------------------------------------------------------ each mechanism alone

ALONE = {
    "wkv": (pz.make_config([(S, pz.wkv_mixer(), None)]), 7),
    "wkv_one_head": (pz.make_config([(S, pz.wkv_mixer(heads=1, dim=24), None)]), 1),
    "wkv_many_small_heads": (pz.make_config([(S, pz.wkv_mixer(heads=12, dim=4), None)]), 16),
    "wkv_rank_33": (pz.make_config([(S, pz.wkv_mixer(heads=3, dim=20), None)]), 33),
    "wkv_rank_72": (pz.make_config([(S, pz.wkv_mixer(heads=2, dim=32), None)]), 72),
    "wkv_rank_130": (pz.make_config([(S, pz.wkv_mixer(heads=2, dim=28), None)]), 130),
    "wkv_heads_of_64": (pz.make_config([(S, pz.wkv_mixer(heads=2, dim=64), None)], width=64), 16),
    "wkv_heads_of_100": (pz.make_config([(S, pz.wkv_mixer(heads=1, dim=100), None)], width=64), 24),
    "wkv_heads_of_130": (pz.make_config([(S, pz.wkv_mixer(heads=2, dim=130), None)], width=64), 8),
    "wkv_heads_of_136": (pz.make_config([(S, pz.wkv_mixer(heads=2, dim=136), None)], width=64), 9),
    "wkv_heads_of_256": (pz.make_config([(S, pz.wkv_mixer(heads=1, dim=256), None)], width=64), 16),
    "wkv_heads_of_300": (pz.make_config([(S, pz.wkv_mixer(heads=1, dim=300), None)], width=64), 8),
    "wkv_heads_of_520": (pz.make_config([(S, pz.wkv_mixer(heads=1, dim=520), None)], width=64), 8),
    "wkv_odd_heads": (pz.make_config([(S, pz.wkv_mixer(heads=3, dim=9), None)], width=37), 5),
    "chunks": (pz.make_config([(A, pz.attn_mixer(), None)]), 7),
    "chunks_of_one": (pz.make_config([(A, pz.attn_mixer(size=1), None)]), 7),
    "chunks_of_two": (pz.make_config([(A, pz.attn_mixer(size=2), None)]), 7),
    "chunks_of_a_page": (pz.make_config([(A, pz.attn_mixer(size=64), None)]), 7),
    "chunks_longer_than_the_sequence": (pz.make_config([(A, pz.attn_mixer(size=4000), None)]), 7),
    "no_chunks": (pz.make_config([(A, pz.attn_mixer(size=0), None)]), 7),
    "one_kv_head": (pz.make_config([(A, pz.attn_mixer(heads=6, kv_heads=1, dim=16, vdim=40, dims=10), None)]), 7),
    "head_per_kv_head": (pz.make_config([(A, pz.attn_mixer(heads=3, kv_heads=3, dim=40, vdim=8, dims=40), None)]), 7),
    "one_pair_turns": (pz.make_config([(A, pz.attn_mixer(dims=2), None)]), 7),
    "all_frequencies_stretched": (pz.make_config([(A, pz.attn_mixer(scaling=(5.0, 40.0, 50.0, 30)), None)]), 7),
    "all_frequencies_kept": (pz.make_config([(A, pz.attn_mixer(scaling=(5.0, 1e-6, 1e-5, 4000)), None)]), 7),
    "all_frequencies_between": (pz.make_config([(A, pz.attn_mixer(base=3.0, scaling=(3.0, 0.5, 60.0, 100)), None)]), 7),
    "heads_of_64": (pz.make_config([(A, pz.attn_mixer(heads=4, kv_heads=1, dim=64, vdim=64, size=50, scale=0.2, dims=32), None)], width=64), 7),
    "heads_of_128": (pz.make_config([(A, pz.attn_mixer(heads=2, kv_heads=2, dim=128, vdim=128, size=37, scale=0.1, dims=128), None)], width=64), 7),
    "keys_wider_than_values": (pz.make_config([(A, pz.attn_mixer(heads=4, kv_heads=2, dim=200, vdim=24, scale=0.07), None)], width=64), 7),
    "values_wider_than_keys": (pz.make_config([(A, pz.attn_mixer(heads=4, kv_heads=4, dim=8, vdim=256, scale=0.4, dims=8), None)], width=64), 7),
    "odd_heads": (pz.make_config([(A, pz.attn_mixer(heads=2, kv_heads=1, dim=9, vdim=13, dims=8), None)]), 7),
    "group_of_20": (pz.make_config([(A, pz.attn_mixer(heads=40, kv_heads=2, dim=8, vdim=24, size=77, dims=8), None)], width=64), 7),
    "a_reader": (pz.make_config([(A, pz.attn_mixer(), None), (A, pz.attn_mixer(heads=4, scale=0.5, kv_from=0), None)]), 7),
    "readers_of_other_chunks": (pz.make_config([(A, pz.attn_mixer(size=21), None), (A, pz.attn_mixer(size=50, kv_from=0), None),
                                                (A, pz.attn_mixer(size=7, kv_from=0), None), (A, pz.attn_mixer(size=0, kv_from=0), None)]), 7),
    "feed_forward": (pz.make_config([(S, pz.wkv_mixer(), pz.dense_mlp(72))]), 7),
    "experts": (pz.make_config([(A, pz.attn_mixer(), MOE())]), 7),
    "no_identity_experts": (pz.make_config([(A, pz.attn_mixer(), MOE(identity=0, experts=6, top=2))]), 7),
    "more_identity_experts": (pz.make_config([(A, pz.attn_mixer(), MOE(identity=9, experts=2, top=4))]), 7),
    "one_expert_each": (pz.make_config([(A, pz.attn_mixer(), MOE(identity=2, experts=40, top=1))]), 7),
    "every_expert": (pz.make_config([(S, pz.wkv_mixer(), MOE(identity=2, experts=3, top=5))]), 7),
    "odd_experts": (pz.make_config([(S, pz.wkv_mixer(), MOE(ff=13, identity=3, experts=5, top=2))], width=45), 7),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ALONE))
def test_mechanism_alone(tmp_path, name, dtype):
    cfg, rank = ALONE[name]
    w = write_model(str(tmp_path), cfg, 3, rank=rank, dtype=dtype)
    ids = prompt(cfg, 141, 5, w)
    ref = pz.forward(cfg, w, ids)
    eng = engine(str(tmp_path), dtype)
    got = whole(eng, ids)
    close(got, ref, dtype, name)
    # and token by token through the cache
    one = in_portions(eng, ids, [1])
    close(one, ref, dtype, name + " token by token")
    same_or_close(one, got, dtype, name + " token by token")


@pytest.mark.parametrize("dtype", DTYPES)
def test_eps_is_read_everywhere(tmp_path, dtype):
    """An eps far from the usual, which every norm of the design shares (embedding, heads, queries and keys, sublayers, last)."""
    layers = [(S, pz.wkv_mixer(), pz.dense_mlp()), (A, pz.attn_mixer(), MOE())]
    cfg = pz.make_config(layers, eps=0.3)
    w = write_model(str(tmp_path), cfg, 4, dtype=dtype)
    ids = prompt(cfg, 60, 2, w)
    ref = pz.forward(cfg, w, ids)
    assert rel_err(pz.forward(pz.make_config(layers, eps=1e-5), w, ids), ref) > 0.05
    eng = engine(str(tmp_path), dtype)
    close(whole(eng, ids), ref, dtype, "prompt")
    close(in_portions(eng, ids, [50, 1]), ref, dtype, "decoding")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompt_through_the_tile_kernels(tmp_path, dtype):
    """A prompt long enough for the prompt kernels' tiles, for many segments of the recurrence and for the experts' tiles."""
    cfg = pz.make_config([(A, pz.attn_mixer(heads=4, kv_heads=2, dim=128, vdim=128, size=260, scale=0.09, dims=64), pz.dense_mlp(256)),
                          (S, pz.wkv_mixer(heads=2, dim=128), MOE(ff=64, experts=5, identity=2, top=2)),
                          (A, pz.attn_mixer(heads=4, kv_heads=2, dim=48, vdim=72, size=333, scale=0.15, dims=32), None),
                          (S, pz.wkv_mixer(heads=3, dim=48), MOE(ff=160, experts=3, identity=1, top=2))], width=64)
    w = write_model(str(tmp_path), cfg, 21, rank=16, dtype=dtype)
    ids = prompt(cfg, 700, 8, w)
    ref = pz.forward(cfg, w, ids)
    eng = engine(str(tmp_path), dtype, max_tokens=2048)
    got = whole(eng, ids)
    close(got, ref, dtype, "700 tokens in one step")
    same_or_close(in_portions(eng, ids, [610, 1]), got, dtype, "the same, its last tokens one by one")
    same_or_close(in_portions(eng, ids, [250, 200, 17, 233]), got, dtype, "long portions")


# ------------------------------------------------------------------ whole models


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_first_tokens_and_one_token(models, name, dtype):
    d, cfg, w = models[name, dtype]
    eng = engine(d, dtype)
    for n in (1, 2, 3):
        ids = prompt(cfg, n, 20 + n, w)
        close(whole(eng, ids), pz.forward(cfg, w, ids), dtype, f"{name} {n} tokens")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_portions_and_decoding(models, name, dtype):
    """Prefill against token-by-token decoding and portions of several sizes, down to two tokens, across page borders,
    chunk edges and the edges of the sixteen-token pieces of the recurrence."""
    d, cfg, w = models[name, dtype]
    ids = prompt(cfg, 200, 13, w)
    layers = []
    ref = pz.forward(cfg, w, ids, layers)
    assert len(layers) == len(cfg["layers"])
    eng = engine(d, dtype)
    base = whole(eng, ids)
    close(base, ref, dtype, name)
    for sizes in ([1], [2], [63, 2, 64, 7], [128, 1], [5, 64, 3], [1, 1, 2, 3, 50], [15, 16, 17, 18, 33]):
        got = in_portions(eng, ids, sizes)
        close(got, ref, dtype, f"{name} portions {sizes}")
        same_or_close(got, base, dtype, f"{name} portions {sizes}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_unequal_batches(models, name, dtype):
    """Requests of different lengths in one batch, then decoded together while the shorter ones end, against each alone."""
    d, cfg, w = models[name, dtype]
    eng = engine(d, dtype, max_tokens=4096)
    lens, extra = [1, 37, 250, 66, 16], [9, 30, 12, 5, 7]
    seqs = [prompt(cfg, n + e, 40 + i, w) for i, (n, e) in enumerate(zip(lens, extra))]
    refs = [pz.forward(cfg, w, s) for s in seqs]
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
        close(g, refs[i], dtype, f"{name} batch, sequence {i}")
        same_or_close(g, alone[i], dtype, f"{name} batch, sequence {i} against itself alone")


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_sequences_at_once(models, dtype):
    """Twenty and seventy single tokens in a step: the products of few rows, of up to 64 and of more."""
    d, cfg, w = models["mixed", dtype]
    eng = engine(d, dtype, max_tokens=16384, max_batch=80)
    for n in (20, 70):
        seqs = [prompt(cfg, 12 + i % 9, 300 + i, w) for i in range(n)]
        slots = [eng.new_sequence() for _ in seqs]
        eng.step([StepItem(s, q[:-3], []) for s, q in zip(slots, seqs)])
        got = [eng.step([StepItem(s, [q[len(q) - 3 + k]], [0]) for s, q in zip(slots, seqs)]).cpu().numpy() for k in range(3)]
        for s in slots:
            eng.end_sequence(s)
        ref = np.stack([pz.forward(cfg, w, q)[-3:] for q in seqs])
        close(np.stack(got, 1).reshape(-1, cfg["vocab"]), ref.reshape(-1, cfg["vocab"]), dtype, f"{n} sequences")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_slots_and_pages_used_again(models, name, dtype):
    """A small cache whose slots and pages go round several times, freed pages poisoned with NaN: a sequence must never
    read a page that it does not hold, and state and the previous token's row start at zero in a slot used before."""
    d, cfg, w = models[name, dtype]
    eng = engine(d, dtype, max_tokens=320, max_batch=3, max_seq_len=256, poison=True)
    for rnd in range(4):
        seqs = [prompt(cfg, n, 70 + 10 * rnd + i, w) for i, n in enumerate((90 + rnd, 33, 70))]
        slots = [eng.new_sequence() for _ in seqs]
        cut = [len(s) // 2 + rnd for s in seqs]
        eng.step([StepItem(slots[i], seqs[i][:cut[i]], []) for i in range(3)])
        eng.end_sequence(slots[1])                        # its slot and pages go to the next sequence at once
        late = prompt(cfg, 40, 90 + rnd, w)
        s_late = eng.new_sequence()
        got_late = eng.step([StepItem(s_late, late, list(range(40)))]).cpu().numpy()
        close(got_late, pz.forward(cfg, w, late), dtype, f"round {rnd}: a sequence in a slot used before")
        for i in (0, 2):
            rest = seqs[i][cut[i]:]
            got = eng.step([StepItem(slots[i], rest, list(range(len(rest))))]).cpu().numpy()
            close(got, pz.forward(cfg, w, seqs[i])[cut[i]:], dtype, f"round {rnd}: sequence {i} continued")
            eng.end_sequence(slots[i])
        eng.end_sequence(s_late)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("own,readers,dims", [(20, [50], (24, 16)), (64, [130, 33], (64, 64)), (33, [0], (16, 16)), (0, [20], (128, 128)), (64, [64], (128, 128))])
def test_a_reader_masks_for_itself(tmp_path, own, readers, dims, dtype):
    """A layer on another layer's keys and values sees what its own mask lets it see, farther or less far than the layer that
    wrote them, in prompts and in decoding, while pages that nobody needs any more are given back (poisoned with NaN)."""
    m = dict(heads=4, kv_heads=2, dim=dims[0], vdim=dims[1], dims=8, scale=0.5 * dims[0] ** -0.5)
    cfg = pz.make_config([(A, pz.attn_mixer(size=own, **m), None)] + [(A, pz.attn_mixer(size=n, kv_from=0, **m), None) for n in readers])
    w = write_model(str(tmp_path), cfg, 9, dtype=dtype)
    ids = prompt(cfg, 230, 3, w)
    ref = pz.forward(cfg, w, ids)
    if readers != [own]:
        alt = json.loads(json.dumps(cfg))
        for layer in alt["layers"][1:]:
            layer["mixer"].pop("mask", None)
            if own:
                layer["mixer"]["mask"] = {"size": own}
        assert rel_err(pz.forward(alt, w, ids), ref) > 0.02, "the reader's own mask does not show"
    for page in (64, 16):
        eng = engine(str(tmp_path), dtype, page_size=page, poison=True)
        close(whole(eng, ids), ref, dtype, "prompt")
        close(in_portions(eng, ids, [130, 1]), ref, dtype, "decoding")
        close(in_portions(eng, ids, [7, 40, 2]), ref, dtype, "portions")


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
    w["embed.norm"][5] = w["embed.norm"][6] = 1.0


def with_chunk(cfg, size):
    c = json.loads(json.dumps(cfg))
    for layer in c["layers"]:
        if layer["type"] == A:
            layer["mixer"]["mask"] = {"size": size}
    return c


def pointed(w, pre, heads, d, q_weight=6.0, k_weight=6.0, noise=0.2):
    """Every query points along its head's last channel (which no rotation touches); a key does so far more than any other
    if its token has the spike."""
    for a in range(heads):
        w[pre + "q"][a * d:(a + 1) * d] *= noise
        w[pre + "q"][(a + 1) * d - 1] = 0.0
        w[pre + "q"][(a + 1) * d - 1, 6] = q_weight
    for g in range(w[pre + "k"].shape[0] // d):
        w[pre + "k"][(g + 1) * d - 1] = 0.0
        w[pre + "k"][(g + 1) * d - 1, 5] = k_weight
    w[pre + "q.norm"][-1] = w[pre + "k.norm"][-1] = 1.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk,page,dims", [(64, 64, (8, 16)), (65, 64, (8, 16)), (63, 64, (8, 12)), (7, 16, (8, 16)), (33, 16, (9, 11)), (2, 64, (8, 16)),
                                             (64, 64, (128, 128)), (65, 64, (128, 128)), (130, 64, (64, 64)), (100, 64, (64, 64)), (150, 64, (16, 64))])
@pytest.mark.parametrize("place", ["first", "last"])
def test_one_key_decides_at_a_chunks_edge(tmp_path, chunk, page, dims, place, dtype):
    """The key of one position stands out for every query that sees it.  At a chunk's first position it decides the whole chunk,
    up to the last position, and nothing after; at a chunk's last position it decides that position alone.  The plain
    implementation with a chunk one longer or shorter must disagree, or the test would show nothing."""
    m = pz.attn_mixer(heads=2, kv_heads=1, dim=dims[0], vdim=dims[1], size=chunk, scale=8.0 / dims[0], dims=4)
    cfg = pz.make_config([(A, m, None)], vocab=50)
    start = max(2, -(-64 // chunk)) * chunk                       # a chunk's first position, not the sequence's
    at = start if place == "first" else start - 1
    ids = crafted_ids(cfg, start + chunk + 40, 3, at)

    def edit(w):
        spike(w)
        pointed(w, "l0.mix.", 2, dims[0])

    w = write_model(str(tmp_path), cfg, 9, edit, dtype=dtype)
    ref = pz.forward(cfg, w, ids)
    lo, hi = max(0, start - 3), min(len(ids), start + chunk + 3)
    for other in (chunk - 1, chunk + 1):
        if other > 0:
            assert rel_err(pz.forward(with_chunk(cfg, other), w, ids)[lo:hi], ref[lo:hi]) > 0.05, "the crafted key does not decide"
    eng = engine(str(tmp_path), dtype, page_size=page)
    assert_close(whole(eng, ids), ref, dtype, f"chunk {chunk}, prompt")
    assert_close(in_portions(eng, ids, [at, 1]), ref, dtype, f"chunk {chunk}, decoding from the key on")
    assert_close(in_portions(eng, ids, [start, 2]), ref, dtype, f"chunk {chunk}, portions from the edge on")
    assert_close(in_portions(eng, ids, [start - 1, 1, chunk - 1, 1, 1, 40]), ref, dtype, f"chunk {chunk}, steps at the edges")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("page,dims", [(64, (16, 24)), (16, (16, 24)), (64, (128, 128)), (64, (64, 64))])
def test_one_far_key_decides_through_another_layers_cache(tmp_path, page, dims, dtype):
    """A key hundreds of positions back, at a page border, decides the second layer, which reads the first one's keys and has no
    mask, while the first layer's chunks are short: in a prompt, in decoding and in portions."""
    m = dict(heads=2, kv_heads=1, dim=dims[0], vdim=dims[1], scale=10.0 / dims[0], dims=4)
    cfg = pz.make_config([(A, pz.attn_mixer(size=20, **m), None), (A, pz.attn_mixer(size=0, kv_from=0, **m), None)], vocab=50)
    far = 63
    ids = crafted_ids(cfg, 330, 3, far)

    def edit(w):
        spike(w)
        pointed(w, "l0.mix.", 2, dims[0])
        for a in range(2):
            q = w["l1.mix.q"]
            q[a * dims[0]:(a + 1) * dims[0]] *= 0.2
            q[(a + 1) * dims[0] - 1] = 0.0
            q[(a + 1) * dims[0] - 1, 6] = 6.0
        w["l1.mix.q.norm"][-1] = 1.0
        w["l0.norm1"][6] = 0.0                            # the constant stays what it is

    w = write_model(str(tmp_path), cfg, 9, edit, dtype=dtype)
    ref = pz.forward(cfg, w, ids)
    alt = pz.forward(cfg, w, ids[:far] + [8] + ids[far + 1:])
    assert rel_err(alt[250:], ref[250:]) > 0.05, "the crafted key does not decide"
    eng = engine(str(tmp_path), dtype, page_size=page, poison=True)
    assert_close(whole(eng, ids), ref, dtype, "prompt")
    assert_close(in_portions(eng, ids, [60, 1]), ref, dtype, "decoding past the key")
    assert_close(in_portions(eng, ids, [far + 1, 2]), ref, dtype, "portions from the key on")
    assert_close(in_portions(eng, ids, [far, 1, 130, 7]), ref, dtype, "the key alone in a step")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dims", [(8, 24), (64, 64), (128, 128)])
def test_the_sink_decides(tmp_path, dims, dtype):
    """Scores far below zero for all keys: nearly all weight goes to the sink, and the head's output is a small part of a
    value, which the norm behind the sublayer leaves small where its eps is not."""
    m = pz.attn_mixer(heads=2, kv_heads=1, dim=dims[0], vdim=dims[1], size=50, scale=4.0 / dims[0], dims=4)
    cfg = pz.make_config([(A, m, None)], vocab=50, eps=1e-2)

    def edit(w):
        w["embed"][:, 6] = 2.0
        w["embed.norm"][6] = 1.0
        pointed(w, "l0.mix.", 2, dims[0], noise=0.1)
        w["l0.mix.k"][:] = 0.1 * np.asarray(w["l0.mix.k"])
        w["l0.mix.k"][-1] = 0.0
        w["l0.mix.k"][-1, 6] = -6.0

    w = write_model(str(tmp_path), cfg, 9, edit, dtype=dtype)
    ids = prompt(cfg, 160, 3, w)
    ref = pz.forward(cfg, w, ids)

    def without(s):
        e = np.exp(s - s.max())
        return e / e.sum()

    with_sink = pz.row_softmax_with_zero_sink
    try:
        pz.row_softmax_with_zero_sink = without
        assert rel_err(pz.forward(cfg, w, ids), ref) > 0.05, "the sink does not decide"
    finally:
        pz.row_softmax_with_zero_sink = with_sink
    eng = engine(str(tmp_path), dtype)
    assert_close(whole(eng, ids), ref, dtype, "prompt")
    assert_close(in_portions(eng, ids, [70, 1]), ref, dtype, "decoding")
    assert_close(in_portions(eng, ids, [2]), ref, dtype, "portions of two")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dims", [(16, 12), (64, 64)])
def test_rotation_and_its_scaling_show(tmp_path, dims, dtype):
    """Sharp attention over rotated channels alone, far from position 0: the plain implementation with another base, another
    factor or without the scaling must disagree."""
    m = pz.attn_mixer(heads=2, kv_heads=2, dim=dims[0], vdim=dims[1], size=0, scale=4.0 * dims[0] ** -0.5, base=30.0, dims=dims[0], scaling=(6.0, 1.0, 8.0, 90))
    cfg = pz.make_config([(A, m, None)], width=64)
    w = write_model(str(tmp_path), cfg, 12, gain=1.0, dtype=dtype)
    ids = prompt(cfg, 230, 4, w)
    ref = pz.forward(cfg, w, ids)
    for edit in (lambda r: r.__setitem__("base", 31.0), lambda r: r.pop("scaling"), lambda r: r["scaling"].__setitem__("factor", 5.0),
                 lambda r: r["scaling"].__setitem__("low", 2.0), lambda r: r["scaling"].__setitem__("high", 6.0), lambda r: r["scaling"].__setitem__("original", 70)):
        alt = json.loads(json.dumps(cfg))
        edit(alt["layers"][0]["mixer"]["rot"])
        assert rel_err(pz.forward(alt, w, ids)[50:], ref[50:]) > 0.01
    eng = engine(str(tmp_path), dtype)
    close(whole(eng, ids), ref, dtype, "prompt")
    close(in_portions(eng, ids, [190, 1]), ref, dtype, "decoding")
    close(in_portions(eng, ids, [39, 2, 41, 64, 3]), ref, dtype, "portions")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim", [(3, 16), (1, 128), (2, 10), (2, 200)])
def test_the_state_remembers_one_early_token(tmp_path, heads, dim, dtype):
    """Decays next to 1 and one token whose key no other token comes near: what it wrote stays in the state, and the
    readings find it hundreds of tokens later, across steps of every size."""
    cfg = pz.make_config([(S, pz.wkv_mixer(heads=heads, dim=dim), None)], vocab=50)
    ids = crafted_ids(cfg, 400, 3, 17)

    def edit(w):
        spike(w)
        x = "l0.mix."
        w[x + "w0"][:] = -9.0
        w[x + "w2"][:] = 0.0
        for s in "rk":
            w[x + "mu." + s][5] = w[x + "mu." + s][6] = 0.0
        w[x + "k"][:, 5] = 0.0
        w[x + "r"] *= 0.1
        for a in range(heads):
            w[x + "k"][a * dim] = 0.0
            w[x + "k"][a * dim, 5] = 4.0                  # channel 0: the spike alone
            w[x + "r"][a * dim] = 0.0
            w[x + "r"][a * dim, 6] = 4.0                  # and the readings' constant
        w[x + "u"][:, 0] = 0.0

    w = write_model(str(tmp_path), cfg, 9, edit, dtype=dtype)
    ref = pz.forward(cfg, w, ids)
    alt = pz.forward(cfg, w, ids[:17] + [8] + ids[18:])
    assert rel_err(alt[350:], ref[350:]) > 0.05, "the early token does not decide"
    eng = engine(str(tmp_path), dtype)
    close(whole(eng, ids), ref, dtype, "prompt")
    close(in_portions(eng, ids, [18, 1]), ref, dtype, "decoding")
    close(in_portions(eng, ids, [17, 1, 100, 2]), ref, dtype, "the token alone in a step")
    close(in_portions(eng, ids, [16, 190, 30]), ref, dtype, "long portions")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("w0", [4.5, 1.5, -9.0, None])
def test_decays_from_nothing_to_everything(tmp_path, w0, dtype):
    """Decays of e^-90 (nothing survives a token, and products of them underflow), of e^-4.5, next to 1, and all of these side by
    side in one head."""
    cfg = pz.make_config([(S, pz.wkv_mixer(heads=2, dim=16), None)])

    def edit(w):
        w["l0.mix.w0"][:] = w0 if w0 is not None else np.tile([4.5, 1.5, -1.0, -9.0], 8)
        w["l0.mix.w2"][:] = 0.2 * np.asarray(w["l0.mix.w2"])

    w = write_model(str(tmp_path), cfg, 9, edit, dtype=dtype)
    ids = prompt(cfg, 210, 6, w)
    ref = pz.forward(cfg, w, ids)
    eng = engine(str(tmp_path), dtype)
    close(whole(eng, ids), ref, dtype, "prompt")
    close(in_portions(eng, ids, [100, 1]), ref, dtype, "decoding")
    close(in_portions(eng, ids, [33, 3, 64]), ref, dtype, "portions")


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_bonus_belongs_to_the_current_token_alone(tmp_path, dtype):
    """A large bonus on one head and none on the other; the plain implementation without it, or with it in the state, must disagree."""
    cfg = pz.make_config([(S, pz.wkv_mixer(heads=2, dim=16), None)])

    def edit(w):
        w["l0.mix.u"][0] = 3.0
        w["l0.mix.u"][1] = 0.0

    w = write_model(str(tmp_path), cfg, 9, edit, dtype=dtype)
    ids = prompt(cfg, 90, 6, w)
    ref = pz.forward(cfg, w, ids)
    alt = dict(w)
    alt["l0.mix.u"] = np.ones_like(w["l0.mix.u"])
    assert rel_err(pz.forward(cfg, alt, ids), ref) > 0.05
    eng = engine(str(tmp_path), dtype)
    close(whole(eng, ids), ref, dtype, "prompt")
    close(in_portions(eng, ids, [40, 1]), ref, dtype, "decoding")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("value", [1.0, 0.0])
def test_blends_of_the_previous_token(tmp_path, value, dtype):
    """Blends that take the previous token's row alone (a sequence's first token then reads zeros), or the token's own alone, whether
    the step is cut between the two or not."""
    cfg = pz.make_config([(S, pz.wkv_mixer(heads=3, dim=12), pz.dense_mlp()), (S, pz.wkv_mixer(heads=2, dim=16), None)])

    def edit(w):
        for k in w:
            if ".mu." in k:
                w[k][:] = value
        for k in ("l0.mix.mu.v", "l1.mix.mu.v"):
            w[k][:] = 0.5                                  # (the first token's output would be empty)
        for k in ("l0.mix.mu.r", "l0.mix.mu.k", "l1.mix.mu.r", "l1.mix.mu.k"):
            w[k][:] = 0.9 * value

    w = write_model(str(tmp_path), cfg, 9, edit, dtype=dtype)
    ids = prompt(cfg, 50, 6, w)
    ref = pz.forward(cfg, w, ids)
    eng = engine(str(tmp_path), dtype)
    for sizes in ([50], [1], [2], [3], [17, 1, 1, 7], [16, 16], [20, 3, 2]):
        close(in_portions(eng, ids, sizes), ref, dtype, f"portions {sizes}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("favoured", ["identity", "tensors", "one", "negative"])
def test_the_correction_decides_the_choice_and_not_the_weights(tmp_path, favoured, dtype):
    """Corrections that send every token to identity experts, to experts with matrices, to one expert of each, and that push every
    choice score below zero."""
    cfg = pz.make_config([(A, pz.attn_mixer(), MOE(ff=40, experts=6, identity=3, top=2))])

    def edit(w):
        c = 0.01 * np.asarray(w["l0.mlp.correction"])
        if favoured == "identity":
            c[6:] += 3.0
        elif favoured == "tensors":
            c[:6] += 3.0
        elif favoured == "one":
            c[2] += 3.0
            c[7] += 3.0
        else:
            c -= 4.0
        w["l0.mlp.correction"] = c

    w = write_model(str(tmp_path), cfg, 9, edit, dtype=dtype)
    ids = prompt(cfg, 300, 6, w)
    ref = pz.forward(cfg, w, ids)
    eng = engine(str(tmp_path), dtype)
    close(whole(eng, ids), ref, dtype, "prompt")
    close(in_portions(eng, ids, [100, 30, 1, 1, 20]), ref, dtype, "portions and single tokens")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(models, dtype):
    """Three hundred tokens one by one behind a short prompt: past several pages and chunks."""
    d, cfg, w = models["mixed", dtype]
    ids = prompt(cfg, 330, 17, w)
    close(in_portions(engine(d, dtype), ids, [30, 1]), pz.forward(cfg, w, ids), dtype, "long decoding")


# ------------------------------------------------------------------ the library's own entry points


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_model_api(models, dtype):
    """Model.generate: the scheduler batches the requests, decodes them together and ends each by itself."""
    d, cfg, w = models["mixed", dtype]
    prompts = [prompt(cfg, n, 50 + n, w) for n in (3, 17, 70, 1)]
    m = Model(ModelConfig(compt_type=dtype, nr_ctx=256, max_tokens=1024))
    m.load(d)
    m.init(top_k=0, top_p=1.0, temp=0.0, repeat_penalty=1.0, repeat_last_n=0, seed=0, end_token=-1)
    got = m.generate(prompts, max_new_tokens=12, stop_ids=[]).tokens
    if dtype == "float32":
        assert got == [pz.greedy_generate(cfg, w, p, 12) for p in prompts]
        return
    # bfloat16 may turn a near-tie: every token the engine chose must be (within rounding) the best continuation of what
    # it had generated so far, by the plain implementation's logits for that very sequence (but for a turned routing)
    for p, g in zip(prompts, got):
        assert len(g) == 12
        lg = pz.forward(cfg, w, p + g)[len(p) - 1:-1]
        gap = lg.max(-1) - lg[np.arange(12), g]
        assert (gap > BF16_TOL * np.abs(lg).max()).sum() <= 1, (g, gap)


def test_command_line(models):
    """bin/llama on a Zeluzen folder: greedy tokens of two requests, float32."""
    d, cfg, w = models["other", "float32"]
    prompts = [prompt(cfg, n, 90 + n, w) for n in (7, 12)]
    want = [pz.greedy_generate(cfg, w, p, 6) for p in prompts]
    args = [os.path.join(ROOT, "bin", "llama"), "-m", d, "-d", "float32", "-c", "128", "-n", "6", "--temp", "0", "--top_k", "0",
            "--top_p", "1", "--repeat_penalty", "1", "-s", "1"]
    for p in prompts:
        args += ["--prompt-ids", ",".join(map(str, p))]
    r = subprocess.run(args, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    got = [[int(t) for t in ln.split(": ")[1].split(",")] for ln in r.stdout.splitlines() if ln.startswith("[")]
    assert got == want


def test_trace_replay_program(models, tmp_path):
    d, cfg, w = models["mixed", "float32"]
    a, b = prompt(cfg, 40, 1, w), prompt(cfg, 9, 2, w)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:33], "want": [0, 32]}, {"id": "b", "tokens": b[:8], "want": [7]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[33:34], "want": [0]}, {"id": "b", "tokens": b[8:], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[34:35], "want": [0]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[35:], "want": [4]}], "end": ["a"]}]
    out = str(tmp_path / "out")
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", out, "--max-tokens", "128"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done %d" % i for i in range(4)]
    ra, rb = pz.forward(cfg, w, a), pz.forward(cfg, w, b)
    V = cfg["vocab"]
    got0 = np.fromfile(os.path.join(out, "0.f32"), "<f4").reshape(-1, V)
    assert_close(got0, np.stack([ra[0], ra[32], rb[7]]), "float32", "step 0")
    assert_close(np.fromfile(os.path.join(out, "1.f32"), "<f4").reshape(-1, V), ra[33:34], "float32", "step 1")
    assert_close(np.fromfile(os.path.join(out, "2.f32"), "<f4").reshape(-1, V), ra[34:35], "float32", "step 2")
    assert_close(np.fromfile(os.path.join(out, "3.f32"), "<f4").reshape(-1, V), ra[39:40], "float32", "step 3")
