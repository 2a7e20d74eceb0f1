"""Layered models (Lasosun) on the GPU against the plain implementation of ``oracle/layered.py``: small random models of many sizes, prompts
whole and in portions, decoding, sessions and batches, and places where a mask, a state or a cache would show."""
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


def floats(bits):
    return {k: mf.bf16_floats(v) for k, v in bits.items()}


def build(tmp_path, config, seed, dtype, bits=None, context=None):
    bits = bits if bits is not None else mf.random_lasosun(config, seed)
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


M, H, A = mf.mamba2, mf.hgrn2, mf.attention
MECHANISMS = {
    "mamba2": ([M(6, 24, 20, groups=3, conv=3, norm_groups=4, ff=72)], 40, 53),            # norm parts cut through heads
    "mamba2 one tap, one group": ([M(3, 40, 32, groups=1, conv=1, norm_groups=1)], 64, 31),
    "mamba2 own groups, wide": ([M(2, 80, 100, groups=2, conv=6, norm_groups=5, ff=130)], 96, 97),
    "mamba2 state beyond the chunked form": ([M(2, 16, 160, groups=1, conv=4, norm_groups=2, ff=24)], 48, 20),
    "hgrn2": ([H(5, 24, 40, ff=56)], 72, 61),
    "hgrn2 one head": ([H(1, 100, 72)], 40, 19),
    "hgrn2 rows beyond the chunked form": ([H(2, 144, 16, ff=40)], 56, 33),
    "attention": ([A(6, 3, 24, 40, 21, 5, ff=48)], 56, 45),
    "attention window 1, block 1": ([A(4, 4, 16, 16, 1, 1)], 32, 29),
    "attention block above window": ([A(8, 1, 40, 20, 6, 11, scale=0.3, ff=64)], 80, 37),
    "attention twelve heads on one": ([A(12, 1, 32, 32, 33, 16)], 64, 41),
    "attention heads of 160": ([A(2, 1, 160, 136, 30, 7, ff=40)], 64, 25),
    "no feed-forward anywhere": ([M(4, 16, 16), A(2, 2, 16, 24, 9, 3), H(2, 16, 16)], 48, 23),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", MECHANISMS)
def test_each_mechanism_whole_in_portions_and_token_by_token(tmp_path, name, dtype):
    layers, width, vocab = MECHANISMS[name]
    config = mf.lasosun_config(layers, width, vocab, 150, eps=3e-5, embed_scale=1.7)
    model, w = build(tmp_path, config, sum(map(ord, name)), dtype)
    ids = ids_for(1, 83, vocab)
    want = plain.lasosun(config, w, ids)
    s = model.new_session()
    check(s.feed(ids, range(len(ids))), want, dtype)
    s.reset()  # the same slot again
    check(in_portions(s, ids, [1]), want, dtype)
    s.reset()
    check(in_portions(s, ids, [2, 9, 31, 3, 16, 8, 1]), want, dtype)
    assert s.position == len(ids)


MIXED = [M(4, 24, 20, groups=2, conv=4, norm_groups=2, ff=88), A(6, 2, 24, 16, 19, 6, ff=88), H(3, 20, 24, ff=40), A(4, 4, 16, 16, 40, 3), M(2, 32, 40, groups=1, conv=2, norm_groups=4), H(2, 40, 16, ff=24)]


def mixed(vocab=71, positions=700, embed_scale=1.0):
    return mf.lasosun_config(MIXED, 56, vocab, positions, eps=1e-5, embed_scale=embed_scale)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_stack_of_all_kinds_in_chunks_of_prefill_and_long_decoding(tmp_path, dtype):
    config = mixed()
    model, w = build(tmp_path, config, 11, dtype)
    ids = ids_for(2, 330, 71)
    want = plain.lasosun(config, w, ids)
    whole = model.new_session()
    check(whole.feed(ids, range(len(ids))), want, dtype)
    s = model.new_session()
    got = np.concatenate([s.feed(ids[:40], range(40)), in_portions(s, ids[40:], [1])])  # the windows pass over decoded tokens many times
    check(got, want, dtype)
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
        before = dec.time_token(1, 5)  # timing a step leaves the sequence as it was
        assert before > 0
        last, _ = dec.forward(int(ids[at]), at)
        check(last[None], want[at:at + 1], dtype)
        with pytest.raises(q.QuintritError) as e:
            dec.forward(3, at - 4)  # a state cannot go back
        assert e.value.code == 6
        last, _ = dec.forward(int(ids[0]), 0)  # but it starts again
        check(last[None], want[:1], dtype)


def needle(window, pool, width=160, vocab=40, seed=5):
    """One attention layer in which the query of token 1 meets the key of token 0 with a score far above all others; token 0's block shows too."""
    config = mf.lasosun_config([A(2, 1, 32, 32, window, pool, scale=1.0)], width, vocab, 400)
    w = floats(mf.random_lasosun(config, seed))
    w["pos"] *= 0.0
    h = plain.rms_norm(w["embed"].astype(np.float64), w["l0.norm1"], config["norm"]["eps"])
    u = np.random.default_rng(seed).normal(0, 1, 32)
    u /= np.linalg.norm(u)
    w["l0.mix.o"] *= 12.0
    w["l0.rg1.b"][:] = 4.0
    w["l0.mix.q"] *= 0.05
    w["l0.mix.k"] *= 0.05
    alpha = (4.5 * pool) ** 0.5 if pool > 1 else 3.0  # a score of 4.5 through the mean of a block
    probe = np.linalg.pinv(h)  # column t answers 1 to token t and 0 to the others
    w["l0.mix.q"] += alpha * np.outer(np.tile(u, 2), probe[:, 1])
    w["l0.mix.k"] += alpha * np.outer(u, probe[:, 0])
    return config, {k: mf.bf16_bits(v) for k, v in w.items()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,pool", [(20, 4), (64, 16), (7, 9), (33, 1)])
def test_keys_just_inside_and_outside_the_window_and_its_blocks(tmp_path, window, pool, dtype):
    config, bits = needle(window, pool)
    model, w = build(tmp_path, config, 5, dtype, bits)
    rng = np.random.default_rng(3)
    shown = 0
    s = model.new_session()
    for base in (0, 1, pool - 1, pool, 30):
        for distance in sorted({1, window - 1, window, window + pool - 1, window + pool, window + 2 * pool, window + 3 * pool + 1, 200}):
            ids = rng.integers(2, 40, base + distance + 1)
            ids[base], ids[-1] = 0, 1
            want = plain.lasosun(config, w, ids)[-1:]
            without = plain.lasosun(config, w, np.where(np.arange(len(ids)) == base, 7, ids))[-1:]
            effect = errors(without, want).max()
            shown += effect > 5 * TOL[dtype]
            for cut in {0, len(ids) - 1, max(0, len(ids) - 9)}:
                s.reset()
                if cut:
                    s.feed(ids[:cut])
                check(s.feed(ids[cut:], [len(ids) - cut - 1]), want, dtype)
    assert shown >= 20  # the needle is seen at many of these distances (and must not be at the others)


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_ring_of_the_cache_is_used_again(tmp_path, dtype):
    """More tokens than the ring holds: old keys are overwritten, their blocks stay visible."""
    config = mf.lasosun_config([A(2, 1, 16, 16, 12, 8)], 32, 30, 2600)
    model, w = build(tmp_path, config, 8, dtype)
    ids = ids_for(4, 2330, 30)
    want = plain.lasosun(config, w, ids)
    s = model.new_session()
    check(s.feed(ids[:2201], range(2000, 2201)), want[2000:2201], dtype)
    check(in_portions(s, ids[2201:], [1, 2, 40, 1, 1]), want[2201:], dtype)
    s.reset()
    check(in_portions(s, ids, [700]), want, dtype)


@pytest.mark.parametrize("kind", ["mamba2", "hgrn2"])
@pytest.mark.parametrize("dtype", DTYPES)
def test_a_state_carries_over_hundreds_of_tokens_and_strong_decays(tmp_path, kind, dtype):
    layer = M(2, 16, 24, groups=1, conv=2, norm_groups=1) if kind == "mamba2" else H(2, 24, 16)
    config = mf.lasosun_config([layer], 40, 30, 600)
    for slow in (True, False):
        w = floats(mf.random_lasosun(config, 9))
        if kind == "mamba2":
            w["l0.mix.A_log"][:] = -9.0 if slow else 3.5      # almost no decay / the state forgotten within a token
        else:
            w["l0.mix.lower"][:] = 0.0
            w["l0.mix.f.b"][:] = 9.0 if slow else -9.0
        w["l0.mix.o"] *= 4.0
        bits = {k: mf.bf16_bits(v) for k, v in w.items()}
        model, w = build(tmp_path, config, 9 + slow, dtype, bits)
        ids = ids_for(6, 400, 30)
        want = plain.lasosun(config, w, ids)
        if slow:  # an early stretch of tokens shows at the end
            other = ids.copy()
            other[:200] = ids_for(7, 200, 30)
            assert errors(plain.lasosun(config, w, other)[-1:], want[-1:]).max() > 2 * TOL[dtype]
        s = model.new_session()
        check(s.feed(ids, range(400)), want, dtype)
        s.reset()
        check(np.concatenate([s.feed(ids[:300], range(300)), in_portions(s, ids[300:], [1])]), want, dtype)


def test_large_products_and_many_tiles_agree_with_32_bit_mode(tmp_path):
    config = mf.lasosun_config([M(16, 64, 128, groups=4, conv=4, norm_groups=4, ff=2048), A(8, 2, 128, 128, 300, 32, ff=2048), H(8, 128, 128, ff=2048)], 1024, 900, 2400)
    ids = ids_for(12, 2300, 900)
    places = list(range(0, 2300, 23)) + [2299]
    bits = mf.random_lasosun(config, 21)
    a, _ = build(tmp_path, config, 21, "bfloat16", bits)
    b, _ = build(tmp_path, config, 21, "float32", bits)
    got, want = a.new_session().feed(ids, places), b.new_session().feed(ids, places)
    check(got, want.astype(np.float64), "bfloat16")
    s = a.new_session()
    s.feed(ids[:2250])
    check(in_portions(s, ids[2250:2260], [1]), b.new_session().feed(ids[:2260], range(2250, 2260)).astype(np.float64), "bfloat16")


def test_batches_of_unequal_sequences_equal_each_alone(tmp_path):
    config = mixed(positions=400)
    model, w = build(tmp_path, config, 13, "bfloat16")
    dec = q.Decoder.open(model.path)
    prompts = [ids_for(20 + i, n, 71) for i, n in enumerate((5, 130, 64, 17, 1))]
    follow = [ids_for(40 + i, 24, 71) for i in range(5)]
    want = [plain.lasosun(config, w, np.concatenate([p, f])) for p, f in zip(prompts, follow)]
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
        row = plain.lasosun(config, w, ids)[-1]
        top = np.sort(row)[-2:]
        margins.append(top[1] - top[0])
        ids.append(int(row.argmax()))
    return ids[len(prompt):], min(margins)


def test_greedy_and_sampled_generation_through_sessions(tmp_path):
    config = mixed(positions=120, embed_scale=0.3)  # (a small embedding: the next token does not just repeat the last)
    model, w = build(tmp_path, config, 16, "float32")
    prompt = ids_for(9, 21, 71)
    want, margin = greedy(config, w, prompt, 30)
    assert margin > 1e-3
    assert model.generate_tokens(prompt, 30).tolist() == want
    s = model.new_session()
    assert s.generate_tokens(prompt, 30).tolist() == want
    assert s.generate_tokens(prompt[:3], 8).tolist() == greedy(config, w, prompt[:3], 8)[0]
    # the sampling loop: top-k 1 and temperature 0 are greedy; equal seeds give equal tokens; the draw follows the device sampler's
    assert s.sample_tokens(prompt, 30, temperature=0.0).tolist() == want
    assert s.sample_tokens(prompt, 30, temperature=1.0, top_k=1).tolist() == want
    one, two = s.sample_tokens(prompt, 20, temperature=1.5, top_k=20, top_p=0.95, seed=7), s.sample_tokens(prompt, 20, temperature=1.5, top_k=20, top_p=0.95, seed=7)
    assert one.tolist() == two.tolist() and one.tolist() != s.sample_tokens(prompt, 20, temperature=1.5, top_k=20, top_p=0.95, seed=0x9E3779B97F4A7C15).tolist()
    fresh = model.new_session()
    row, state = fresh.feed(prompt, [len(prompt) - 1])[0], 7
    for t in one:
        tok, state = q.sample_logits(row, 1.5, 20, 0.95, state)
        assert tok == t
        row = fresh.feed([tok], [0])[0]
    with pytest.raises(q.QuintritError) as e:
        s.feed(list(range(60)) * 3, keep_context=False)
    assert e.value.code == 11
    with pytest.raises(q.QuintritError) as e:
        model.generate("text", 3)  # the folder has no tokenizer
    assert e.value.code == 6
    # the command line
    r = subprocess.run([sys.executable, "-m", "quintrit_b200.generate", "--model", model.path, "--dtype", "float32", "--tokens", ",".join(map(str, prompt)), "--max-new", "30"],
                       capture_output=True, text=True, cwd=q.library_path().rsplit("/quintrit_b200/", 1)[0])
    assert r.returncode == 0 and [int(x) for x in r.stdout.split(",")] == want, r.stderr


def test_trace_replay(tmp_path):
    config = mixed(positions=200)
    model, w = build(tmp_path, config, 15, "float32")
    a, b = ids_for(1, 40, 71), ids_for(2, 33, 71)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:25].tolist(), "want": [24, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b.tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[25:].tolist(), "want": [0, 14]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "c", "tokens": b[:2].tolist(), "want": [0, 1]}], "end": ["b", "c"]}]
    root = q.library_path().rsplit("/quintrit_b200/", 1)[0]
    r = subprocess.run([sys.executable, f"{root}/bin/trace_run", "--model", model.path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "100"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    wa, wb = plain.lasosun(config, w, a), plain.lasosun(config, w, b)
    for step, want in ((0, wa[[24, 3]]), (2, wa[[25, 39]]), (3, wb[[0, 1]])):
        check(np.fromfile(tmp_path / f"{step}.f32", "<f4").reshape(-1, 71), want, "float32")
    assert not (tmp_path / "1.f32").exists()
