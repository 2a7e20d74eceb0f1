"""Tosevik on the GPU against the plain implementation of ``oracle/layered.py``: small random models of many sizes, prompts whole and in portions,
decoding, sessions and batches, and places where a key, a state, a decay, a chosen expert or a cache row would show."""
import json
import subprocess
import sys

import numpy as np
import pytest

import quintrit_b200 as q
from oracle import layered as plain
from quintrit_b200 import model_folder as mf
from quintrit_b200.runtime import Model

pytestmark = pytest.mark.gpu

TOL = {"float32": 4e-5, "bfloat16": 5e-2}  # RMS error of a position's logits over the RMS of all logits
DTYPES = list(TOL)
CODE = 12  # dimensions of the residual stream that carry a token's routing (see settled)


def floats(bits):
    return {k: mf.bf16_floats(v) for k, v in bits.items()}


def call(z, c):
    """The smallest gap (of logits) between a chosen and a passed-over group or expert."""
    gaps, groups = [1e9], z.reshape(c["groups"]["count"], -1).max(1)
    order, keep = np.sort(groups)[::-1], c["groups"]["keep"]
    if keep < len(order):
        gaps.append(order[keep - 1] - order[keep])
    allowed = np.sort(np.where(np.repeat(groups >= order[keep - 1], len(z) // len(groups)), z, -np.inf))[::-1]
    if c["top"] < np.isfinite(allowed).sum():
        gaps.append(allowed[c["top"] - 1] - allowed[c["top"]])
    return min(gaps)


def settled(config, w, seed=0):
    """Makes the choice of experts a clear one, so that rounding cannot change it: a few dimensions of the residual stream hold one of six patterns
    of signs that only the embedding writes, the routers read little else, and tell the patterns apart well."""
    rng = np.random.default_rng(seed + 1000)
    codes = rng.choice([-1.0, 1.0], (6, CODE))
    w["embed"][:, :CODE] = 2.0 * codes[np.arange(config["vocab"]) % 6]
    for name, a in w.items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("o", "down"):
            a[:CODE] = 0.0
        elif leaf == "norm2" or name == "embed.norm":
            a[:CODE], w[name + ".b"][:CODE] = 1.0, 0.0
        elif leaf == "router":
            c = config["layers"][int(name[1:name.index(".")])]["mlp"]["router"]
            tries = rng.normal(0, 1.0, (400, len(a), CODE))
            a[:, CODE:] *= 0.02
            a[:, :CODE] = max(tries, key=lambda r: min(call(r @ s, c) for s in codes))
    return w


def settled_bits(config, seed):
    return {k: mf.bf16_bits(v) for k, v in settled(config, floats(mf.random_tosevik(config, seed)), seed).items()}


def margin(config, w, ids):
    """The closest call of any router: the smallest gap (of logits) between a chosen and a passed-over expert or group."""
    gaps, route = [], plain.route

    def watched(z, c):
        gaps.append(call(z, c))
        return route(z, c)

    plain.route = watched
    try:
        logits = plain.tosevik(config, w, ids)
    finally:
        plain.route = route
    return min(gaps, default=1.0), logits


def build(tmp_path, config, seed, dtype, bits=None, context=None):
    bits = bits if bits is not None else settled_bits(config, seed) if dtype == "bfloat16" else mf.random_tosevik(config, seed)
    path = mf.write_folder(str(tmp_path / f"m{seed}_{dtype}"), config, bits)
    return Model.load(path, dtype=dtype, context=context), floats(bits)


def ids_for(seed, n, vocab):
    return np.random.default_rng(seed).integers(0, vocab, n)


def errors(got, want):
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((w * w).mean())


def check(got, want, dtype):
    e = errors(got, want)
    assert e.max() < TOL[dtype], f"position {int(e.argmax())}: {e.max():.2e}"


def in_portions(session, ids, sizes):
    """Feeds ids in portions of the given sizes in turn; logits of every position."""
    out, at, k = [], 0, 0
    while at < len(ids):
        n = min(sizes[k % len(sizes)], len(ids) - at)
        out.append(session.feed(ids[at:at + n], range(n)))
        at, k = at + n, k + 1
    return np.concatenate(out)


R, A, E, RL, PL = mf.retention, mf.logistic, mf.experts, mf.retention_layer, mf.parallel_layer
MECHANISMS = {
    "retention": ([RL(R(5, 24, 40), E(8, 3, 40, 72))], 72, 61),
    "retention, part of a head rotated": ([RL(R(3, 40, 24, rot=10, base=300.0), E(8, 2, 24, 24, 4, 2, 1.3))], 64, 53),
    "retention, odd sizes": ([RL(R(1, 18, 33, decay=[0.9]), E(6, 6, 17, 9))], 50, 29),
    "retention, wide heads": ([RL(R(2, 100, 160, rot=64), E(4, 1, 130, 40, 2, 1))], 96, 47),
    "retention, state rows beyond 128": ([RL(R(2, 144, 200), E(4, 2, 64, 64))], 80, 31),
    "retention, values beyond the chunked form": ([RL(R(2, 16, 272), E(4, 2, 64, 64))], 80, 31),
    "retention without feed-forward": ([RL(R(4, 16, 16))], 48, 23),
    "side by side": ([PL(A(6, 3, 24, 40, every=17), R(4, 16, 24), E(9, 2, 40, 56, 3, 2))], 56, 45),
    "side by side, one kv head": ([PL(A(8, 1, 40, 20, coef=1.1, every=5, scale=0.3), R(2, 32, 16), E(10, 4, 48, 24, 5, 3, 0.7))], 80, 37),
    "side by side, twelve heads on one": ([PL(A(12, 1, 32, 32), R(1, 64, 64), E(4, 2, 32, 32))], 64, 41),
    "side by side, a kv head each": ([PL(A(5, 5, 16, 48, coef=0.0), R(3, 8, 8), E(4, 2, 32, 32, 4, 2))], 64, 41),
    "side by side, heads of 160 and 136": ([PL(A(2, 1, 160, 136), R(2, 24, 24), E(4, 2, 32, 32))], 64, 25),
    "side by side, heads of 250": ([PL(A(2, 2, 250, 70), R(2, 24, 24))], 64, 25),
    "side by side, small odd heads": ([PL(A(3, 1, 5, 7, every=1), R(2, 6, 5), E(33, 5, 12, 20, 11, 4))], 40, 21),
    "many groups, most dropped": ([RL(R(2, 16, 16), E(80, 2, 16, 16, 40, 3))], 64, 50),
    "every expert": ([RL(R(2, 16, 16), E(3, 3, 16, 16, 1, 1, 2.5))], 64, 50),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", MECHANISMS)
def test_each_mechanism_whole_in_portions_and_token_by_token(tmp_path, name, dtype):
    layers, width, vocab = MECHANISMS[name]
    config = mf.tosevik_config(layers, width, vocab, eps=3e-5)
    model, w = build(tmp_path, config, sum(map(ord, name)), dtype)
    ids = ids_for(1, 147, vocab)
    clear, want = margin(config, w, ids)
    assert clear > (0.02 if dtype == "bfloat16" else 1e-5)
    s = model.new_session()
    check(s.feed(ids, range(len(ids))), want, dtype)
    s.reset()  # the same slot again
    check(in_portions(s, ids, [1]), want, dtype)
    s.reset()
    check(in_portions(s, ids, [2, 9, 31, 3, 16, 8, 1, 64]), want, dtype)
    assert s.position == len(ids)


MIXED = [RL(R(4, 24, 20), E(8, 3, 40, 72, 4, 2, 1.4)), PL(A(6, 2, 24, 16, every=19), R(3, 20, 24), E(8, 2, 24, 40)), PL(A(4, 4, 16, 16), R(2, 40, 16)), RL(R(2, 32, 40, rot=16)),
         RL(R(2, 16, 64), E(12, 4, 16, 24, 3, 2, 0.8))]


def mixed(vocab=71):
    return mf.tosevik_config(MIXED, 56, vocab, eps=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_stack_of_all_kinds_in_chunks_of_prefill_and_long_decoding(tmp_path, dtype):
    config = mixed()
    model, w = build(tmp_path, config, 11, dtype)
    ids = ids_for(2, 330, 71)
    clear, want = margin(config, w, ids)
    assert clear > (0.02 if dtype == "bfloat16" else 1e-5)
    check(model.new_session().feed(ids, range(len(ids))), want, dtype)
    s = model.new_session()
    check(np.concatenate([s.feed(ids[:40], range(40)), in_portions(s, ids[40:], [1])]), want, dtype)
    s.reset()
    check(in_portions(s, ids, [64, 2, 100, 5, 17]), want, dtype)
    # the same through the decoder handle, where portions below eight tokens are chunks too
    dec = q.Decoder.open(model.path) if dtype == "bfloat16" else None
    if dec is not None:
        at = 0
        for n in (2, 3, 30, 2, 7, 1, 60, 4):
            last, nxt = dec.prefill(ids[at:at + n], at)
            at += n
            check(last[None], want[at - 1:at], dtype)
            assert nxt == int(np.argmax(last))
        assert dec.time_token(1, 5) > 0  # timing a step leaves the sequence as it was
        last, _ = dec.forward(int(ids[at]), at)
        check(last[None], want[at:at + 1], dtype)
        with pytest.raises(q.QuintritError) as e:
            dec.forward(3, at - 4)  # a state cannot go back
        assert e.value.code == 6
        last, _ = dec.forward(int(ids[0]), 0)  # but it starts again
        check(last[None], want[:1], dtype)


def needle(seed=5, heads=4, dim=32, width=160, vocab=40, temp=0.0):
    """One layer whose attention alone reaches the output, in which the query of token 1 meets the key of token 0 and no other: every other weight
    is that of a low bias. The slope of the head that shows it is small (the last of many)."""
    config = mf.tosevik_config([PL(A(heads, 1, dim, dim, coef=temp, every=50, scale=1.0), R(1, 8, 8))], width, vocab)
    w = floats(mf.random_tosevik(config, seed))
    w["l0.mix.right.out"][:] = 0.0
    w["l0.mix.left.out"][:] = 3.0
    w["l0.mix.left.pb"][:] = -14.0
    w["l0.mix.left.q.norm"][:] = 1.0
    w["l0.mix.left.k.norm"][:] = 1.0
    h = plain.dynamic_tanh(plain.dynamic_tanh(w["embed"].astype(np.float64), w["embed.norm"], w["embed.norm.b"], w["embed.norm.alpha"]), w["l0.norm1"], w["l0.norm1.b"], w["l0.norm1.alpha"])
    u = np.random.default_rng(seed).normal(0, 1, dim)
    u /= np.linalg.norm(u)
    probe = np.linalg.pinv(h)  # column t answers 1 to token t and 0 to the others
    w["l0.mix.left.q"] += 40.0 * np.outer(np.tile(u, heads), probe[:, 1])
    w["l0.mix.left.k"] += 40.0 * np.outer(u, probe[:, 0])
    return config, {k: mf.bf16_bits(v) for k, v in w.items()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("temp", [0.0, 0.25])
def test_one_key_far_back_and_at_the_borders_of_tiles_and_shares(tmp_path, temp, dtype):
    config, bits = needle(temp=temp)
    model, w = build(tmp_path, config, 5, dtype, bits)
    rng = np.random.default_rng(3)
    shown = 0
    s = model.new_session()
    for base in (0, 1, 63, 64, 127, 128, 200):
        for distance in (1, 2, 48, 49, 62, 63, 64, 65, 127, 128, 129, 191, 300, 511):
            ids = rng.integers(2, 40, base + distance + 1)
            ids[base], ids[-1] = 0, 1
            want = plain.tosevik(config, w, ids)[-1:]
            without = plain.tosevik(config, w, np.where(np.arange(len(ids)) == base, 7, ids))[-1:]
            shown += errors(without, want).max() > 5 * TOL[dtype]
            for cut in {0, len(ids) - 1, max(0, len(ids) - 9)}:
                s.reset()
                if cut:
                    s.feed(ids[:cut])
                check(s.feed(ids[cut:], [len(ids) - cut - 1]), want, dtype)
    assert shown >= 90  # the needle is seen at nearly all of these distances


@pytest.mark.parametrize("dtype", DTYPES)
def test_distance_slopes_and_biases_of_every_head(tmp_path, dtype):
    """Queries and keys that all agree: the weights follow the distance alone, head by head."""
    config = mf.tosevik_config([PL(A(6, 2, 16, 24, coef=0.0, scale=0.01), R(1, 8, 8))], 64, 30)
    w = floats(mf.random_tosevik(config, 4))
    w["l0.mix.right.out"][:] = 0.0
    w["l0.mix.left.out"] *= 3.0
    w["l0.mix.left.pb"][:] = [3.0, -2.0, 1.0, 0.0, 4.0, -5.0]
    model, w = build(tmp_path, config, 4, dtype, {k: mf.bf16_bits(v) for k, v in w.items()})
    ids = ids_for(4, 300, 30)
    want = plain.tosevik(config, w, ids)
    s = model.new_session()
    check(s.feed(ids, range(300)), want, dtype)
    s.reset()
    check(in_portions(s, ids, [150, 1, 1, 1, 70]), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_query_temperature_steps_where_it_should(tmp_path, dtype):
    config = mf.tosevik_config([PL(A(2, 2, 16, 16, coef=6.0, every=23, scale=0.6), R(1, 8, 8))], 64, 30)
    w = floats(mf.random_tosevik(config, 8))
    w["l0.mix.right.out"][:] = 0.0
    w["l0.mix.left.out"] *= 3.0
    model, w = build(tmp_path, config, 8, dtype, {k: mf.bf16_bits(v) for k, v in w.items()})
    ids = ids_for(5, 100, 30)
    want = plain.tosevik(config, w, ids)
    assert plain.query_temperature([21, 22, 45, 46], 6.0, 23)[[0, 1]].tolist() == [1.0, 1.0 + 6.0 * np.log(2.0)]
    other = json.loads(json.dumps(config))
    other["layers"][0]["mixer"]["left"]["q_temp"]["every"] = 24
    assert errors(plain.tosevik(other, w, ids), want)[[22, 45]].min() > 2 * TOL[dtype]
    s = model.new_session()
    check(s.feed(ids, range(100)), want, dtype)
    s.reset()
    check(in_portions(s, ids, [1]), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decay", [[1.0, 0.999], [0.5, 0.02], [0.0, 0.97]])
def test_a_state_carries_over_hundreds_of_tokens_and_strong_decays(tmp_path, decay, dtype):
    config = mf.tosevik_config([RL(R(2, 24, 16, decay=decay))], 40, 30)
    w = floats(mf.random_tosevik(config, 9))
    w["l0.mix.o"] *= 4.0
    model, w = build(tmp_path, config, 9, dtype, {k: mf.bf16_bits(v) for k, v in w.items()})
    ids = ids_for(6, 400, 30)
    want = plain.tosevik(config, w, ids)
    if decay[0] == 1.0:  # an early stretch of tokens shows at the end
        other = ids.copy()
        other[:200] = ids_for(7, 200, 30)
        assert errors(plain.tosevik(config, w, other)[-1:], want[-1:]).max() > 2 * TOL[dtype]
    s = model.new_session()
    check(s.feed(ids, range(400)), want, dtype)
    s.reset()
    check(np.concatenate([s.feed(ids[:300], range(300)), in_portions(s, ids[300:], [1])]), want, dtype)
    for sizes in ([64], [63, 65], [128, 2], [65, 62]):  # a chunk of the recurrence is 64 tokens of a portion
        s.reset()
        check(in_portions(s, ids, sizes), want, dtype)


def lone_memory():
    """A retention layer in which little but token 0 writes to the state, and token 1 reads it."""
    config = mf.tosevik_config([RL(R(1, 16, 16, decay=[0.9995], base=50.0))], 96, 40)
    w = floats(mf.random_tosevik(config, 12))
    h = plain.dynamic_tanh(plain.dynamic_tanh(w["embed"].astype(np.float64), w["embed.norm"], w["embed.norm.b"], w["embed.norm.alpha"]), w["l0.norm1"], w["l0.norm1.b"], w["l0.norm1.alpha"])
    probe = np.linalg.pinv(h)
    u = np.random.default_rng(1).normal(0, 1, 16)
    w["l0.mix.k"] = w["l0.mix.k"] * 0.01 + 20.0 * np.outer(u, probe[:, 0])
    w["l0.mix.q"] = w["l0.mix.q"] * 0.01 + np.outer(u, probe[:, 1])
    w["l0.mix.o"] *= 3.0
    return config, {k: mf.bf16_bits(v) for k, v in w.items()}


@pytest.mark.parametrize("dtype", DTYPES)
def test_one_memory_read_at_the_edges_of_chunks(tmp_path, dtype):
    config, bits = lone_memory()
    model, w = build(tmp_path, config, 12, dtype, bits)
    rng = np.random.default_rng(8)
    s = model.new_session()
    for base in (0, 1, 62, 63, 64, 65, 130):
        for gap in (1, 62, 63, 64, 65, 127, 128, 129, 260):
            ids = rng.integers(2, 40, base + gap + 1)
            ids[base], ids[-1] = 0, 1
            want = plain.tosevik(config, w, ids)[-1:]
            for cut in {0, len(ids) - 1, max(0, len(ids) - 9), (len(ids) // 2)}:
                s.reset()
                if cut:
                    s.feed(ids[:cut])
                check(s.feed(ids[cut:], [len(ids) - cut - 1]), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_experts_with_all_tokens_none_and_more_than_a_tile(tmp_path, dtype):
    """Ids that share a pattern of signs (settled) all go to the same few experts; then ids that spread."""
    config = mf.tosevik_config([RL(R(2, 16, 16), E(16, 3, 72, 24, 4, 2, 12.0)), RL(R(2, 16, 16), E(5, 2, 200, 100, scale=3.0))], 72, 30)
    model, w = build(tmp_path, config, 14, dtype)
    s = model.new_session()
    for ids in (3 + 6 * ids_for(1, 421, 5), np.repeat([2, 4], 150) + 6 * ids_for(2, 300, 4), ids_for(3, 290, 30)):
        clear, want = margin(config, w, ids)
        assert clear > (0.02 if dtype == "bfloat16" else 1e-5)
        s.reset()
        check(s.feed(ids, range(len(ids))), want, dtype)
    # the restriction to the best groups decides something
    free = json.loads(json.dumps(config))
    free["layers"][0]["mlp"]["router"]["groups"] = {"count": 1, "keep": 1}
    assert errors(plain.tosevik(free, w, ids), want).max() > 3 * TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_prompt_longer_than_a_pass_and_a_cache_filled_to_its_end(tmp_path, dtype):
    config = mf.tosevik_config([PL(A(2, 1, 16, 16), R(2, 16, 16), E(4, 2, 16, 16))], 32, 30)
    model, w = build(tmp_path, config, 8, dtype, context=2330)
    ids = ids_for(4, 2330, 30)
    want = plain.tosevik(config, w, ids)
    s = model.new_session()
    check(s.feed(ids[:2201], range(2000, 2201)), want[2000:2201], dtype)
    check(in_portions(s, ids[2201:], [1, 2, 40, 1, 1]), want[2201:], dtype)
    with pytest.raises(q.QuintritError) as e:
        s.feed([1])
    assert e.value.code == 11
    s.reset()
    check(in_portions(s, ids, [700]), want, dtype)


def test_large_products_and_many_tiles_agree_with_32_bit_mode(tmp_path):
    config = mf.tosevik_config([RL(R(8, 64, 128), E(16, 4, 512, 1024, 4, 2)), PL(A(8, 2, 128, 128), R(4, 128, 256), E(16, 4, 512, 1024))], 1024, 900)
    ids = ids_for(12, 2300, 900)
    places = list(range(0, 2300, 23)) + [2299]
    bits = settled_bits(config, 21)
    a, _ = build(tmp_path, config, 21, "bfloat16", bits)
    b, _ = build(tmp_path, config, 21, "float32", bits)
    got, want = a.new_session().feed(ids, places), b.new_session().feed(ids, places)
    check(got, want.astype(np.float64), "bfloat16")
    s = a.new_session()
    s.feed(ids[:2250])
    check(in_portions(s, ids[2250:2260], [1]), b.new_session().feed(ids[:2260], range(2250, 2260)).astype(np.float64), "bfloat16")


def test_batches_of_unequal_sequences_equal_each_alone(tmp_path):
    config = mixed()
    model, w = build(tmp_path, config, 11, "bfloat16")
    dec = q.Decoder.open(model.path, context=400)
    prompts = [ids_for(20 + i, n, 71) for i, n in enumerate((5, 130, 64, 17, 1))]
    follow = [ids_for(40 + i, 24, 71) for i in range(5)]
    want = []
    for p, f in zip(prompts, follow):
        clear, logits = margin(config, w, np.concatenate([p, f]))
        assert clear > 0.02
        want.append(logits)
    batch = q.Batch(dec, 5)
    for turn in range(2):  # the second turn uses every slot again
        for i in (3, 0, 4, 1, 2):
            batch.rewind(i, 0)
            last, _ = batch.prefill(i, prompts[i])
            check(last[None], want[i][len(prompts[i]) - 1:len(prompts[i])], "bfloat16")
        at = [0] * 5
        for step in range(12):
            order = [[0, 1, 2, 3, 4], [4, 2, 0], [1, 3]][step % 3]
            chosen, logits = batch.step(order, [int(follow[i][at[i]]) for i in order], want_logits=True)
            for z, i in enumerate(order):
                check(logits[z][None], want[i][len(prompts[i]) + at[i]][None], "bfloat16")
                assert chosen[z] == int(np.argmax(logits[z]))
                at[i] += 1
    with pytest.raises(q.QuintritError):
        batch.rewind(0, 3)
    batch.free()


def greedy(config, w, prompt, n):
    ids, margins = list(prompt), []
    for _ in range(n):
        row = plain.tosevik(config, w, ids)[-1]
        top = np.sort(row)[-2:]
        margins.append(top[1] - top[0])
        ids.append(int(row.argmax()))
    return ids[len(prompt):], min(margins)


def test_greedy_and_sampled_generation_through_sessions(tmp_path):
    config = mixed()
    model, w = build(tmp_path, config, 16, "float32", context=120)
    prompt = ids_for(9, 21, 71)
    want, clear = greedy(config, w, prompt, 30)
    assert clear > 1e-4
    assert model.generate_tokens(prompt, 30).tolist() == want
    s = model.new_session()
    assert s.generate_tokens(prompt, 30).tolist() == want
    assert s.generate_tokens(prompt[:3], 8).tolist() == greedy(config, w, prompt[:3], 8)[0]
    assert s.sample_tokens(prompt, 30, temperature=0.0).tolist() == want
    assert s.sample_tokens(prompt, 30, temperature=1.0, top_k=1).tolist() == want
    one, two = s.sample_tokens(prompt, 20, temperature=1.5, top_k=20, top_p=0.95, seed=7), s.sample_tokens(prompt, 20, temperature=1.5, top_k=20, top_p=0.95, seed=7)
    assert one.tolist() == two.tolist()
    fresh = model.new_session()
    row, state = fresh.feed(prompt, [len(prompt) - 1])[0], 7
    for t in one:
        tok, state = q.sample_logits(row, 1.5, 20, 0.95, state)
        assert tok == t
        row = fresh.feed([tok], [0])[0]
    with pytest.raises(q.QuintritError) as e:
        s.feed(list(range(60)) * 3, keep_context=False)
    assert e.value.code == 11
    r = subprocess.run([sys.executable, "-m", "quintrit_b200.generate", "--model", model.path, "--dtype", "float32", "--tokens", ",".join(map(str, prompt)), "--max-new", "30"],
                       capture_output=True, text=True, cwd=q.library_path().rsplit("/quintrit_b200/", 1)[0])
    assert r.returncode == 0 and [int(x) for x in r.stdout.split(",")] == want, r.stderr


def test_trace_replay(tmp_path):
    config = mixed()
    model, w = build(tmp_path, config, 15, "float32")
    a, b = ids_for(1, 40, 71), ids_for(2, 33, 71)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:25].tolist(), "want": [24, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b.tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[25:].tolist(), "want": [0, 14]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "c", "tokens": b[:2].tolist(), "want": [0, 1]}], "end": ["b", "c"]}]
    root = q.library_path().rsplit("/quintrit_b200/", 1)[0]
    for most in ("100", "0"):
        r = subprocess.run([sys.executable, f"{root}/bin/trace_run", "--model", model.path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", most],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True)
        assert r.returncode == 0, r.stderr
        assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
        wa, wb = plain.tosevik(config, w, a), plain.tosevik(config, w, b)
        for step, want in ((0, wa[[24, 3]]), (2, wa[[25, 39]]), (3, wb[[0, 1]])):
            check(np.fromfile(tmp_path / f"{step}.f32", "<f4").reshape(-1, 71), want, "float32")
        assert not (tmp_path / "1.f32").exists()
