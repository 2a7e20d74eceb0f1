"""Tosevik without a GPU: the reader (config.json, tensors, what it refuses), and the plain implementation against other ways of writing the same
equations."""
import json
import os

import numpy as np
import pytest

import quintrit_b200 as q
from oracle import layered as plain
from quintrit_b200 import model_folder as mf

LAYERS = [mf.retention_layer(mf.retention(3, 12, 20, rot=8, base=5000.0), mf.experts(8, 3, 24, 40, groups=4, keep=2, scale=1.25)),
          mf.parallel_layer(mf.logistic(4, 2, 16, 24, coef=0.4, every=10, scale=0.3), mf.retention(2, 8, 16, decay=[0.5, 0.875])),
          mf.retention_layer(mf.retention(1, 16, 8), mf.experts(5, 1, 16, 8))]


def config(layers=LAYERS, width=28, vocab=19, eps=2e-5):
    return mf.tosevik_config(layers, width, vocab, eps)


def folder(tmp_path, cfg=None, tensors=None, name="m"):
    cfg = cfg or config()
    return mf.write_folder(str(tmp_path / name), cfg, tensors if tensors is not None else mf.random_tosevik(cfg, 1))


def test_describe_reads_every_size_and_constant(tmp_path):
    d = q.gguf_describe(folder(tmp_path))
    assert (d["architecture"], d["vocab_size"], d["hidden_size"], d["num_layers"], d["context_length"], d["tied"]) == ("Tosevik", "19", "28", "3", "0", "0")
    assert float(d["rms_norm_eps"]) == pytest.approx(2e-5)
    assert d["layer_0"].startswith("retention heads=3 vdim=20 dim=12 rot=8/5000 decay=0.96875,")
    assert d["layer_0"].endswith(" ff=24 experts=8 top=3 groups=2/4 router_scale=1.25 shared_ff=40")
    left, right = d["layer_1"].split(" | ")
    assert left.startswith("logistic_attention heads=4 vdim=24 dim=16 kv_heads=2 scale=0.3") and "q_temp=0.4" in left and left.endswith("/10")
    assert right == "retention heads=2 vdim=16 dim=8 rot=8/10000 decay=0.5,0.875 ff=0"
    assert d["layer_2"].endswith("ff=16 experts=5 top=1 groups=1/1 router_scale=1 shared_ff=8")
    assert {t["name"]: t["shape"] for t in d["tensors"]} == {k: tuple(v) for k, v in mf.tosevik_shapes(config()).items()}


def test_parts_that_may_be_left_out(tmp_path):
    cfg = config([mf.retention_layer(mf.retention(2, 8, 8), mf.experts(4, 2, 8, 8)), mf.parallel_layer(mf.logistic(2, 1, 8, 8), mf.retention(2, 8, 8))])
    tensors = mf.random_tosevik(cfg, 1)
    del cfg["layers"][0]["mixer"]["rot"], cfg["layers"][0]["mlp"]["router"]["groups"]
    cfg["layers"][1]["mixer"]["left"]["q_temp"] = None
    d = q.gguf_describe(folder(tmp_path, cfg, tensors))
    assert "rot=0/" in d["layer_0"] and "groups=1/1" in d["layer_0"] and "q_temp=0/1 " in d["layer_1"]


def refused(path, code, text=""):
    with pytest.raises(q.QuintritError) as e:
        q.gguf_describe(path)
    assert e.value.code == code and text in str(e.value), str(e.value)


def test_config_mistakes_are_named(tmp_path):
    good = config()
    tensors = mf.random_tosevik(good, 1)

    def variant(name, change):
        c = json.loads(json.dumps(good))
        change(c)
        return folder(tmp_path, c, tensors, name)

    L = lambda c, i: c["layers"][i]
    refused(variant("a", lambda c: c.pop("norm")), 10, "norm")
    refused(variant("b", lambda c: L(c, 0)["mixer"].pop("dim")), 10, "layers[0].mixer.dim")
    refused(variant("c", lambda c: L(c, 0)["mixer"].update(decay=[0.5, 0.5])), 10, "decay")
    refused(variant("d", lambda c: L(c, 0)["mixer"].update(decay=[0.5, 0.5, 1.5])), 10, "decay")
    refused(variant("e", lambda c: L(c, 0)["mixer"]["rot"].update(dims=7)), 6, "rot.dims")
    refused(variant("f", lambda c: L(c, 0)["mixer"]["rot"].update(dims=14)), 6, "rot.dims")
    refused(variant("g", lambda c: L(c, 1)["mixer"].pop("right")), 10, "right")
    refused(variant("h", lambda c: L(c, 1)["mixer"]["left"].update(kv_heads=3)), 6, "kv_heads")
    refused(variant("i", lambda c: L(c, 1)["mixer"]["left"].pop("scale")), 10, "left.scale")
    refused(variant("j", lambda c: L(c, 1)["mixer"]["left"]["q_temp"].update(every=0)), 10, "q_temp.every")
    refused(variant("k", lambda c: L(c, 2).update(type="gla")), 10, "gla")
    refused(variant("l", lambda c: L(c, 0)["mlp"].update(kind="dense")), 10, "dense")
    refused(variant("m", lambda c: L(c, 0)["mlp"]["router"]["groups"].update(count=3)), 6, "groups.count")
    refused(variant("n", lambda c: L(c, 0)["mlp"]["router"]["groups"].update(keep=5)), 6, "groups.keep")
    refused(variant("o", lambda c: L(c, 0)["mlp"]["router"].update(top=5)), 6, "top")
    refused(variant("p", lambda c: L(c, 0)["mlp"].pop("shared")), 10, "shared")
    refused(variant("q", lambda c: L(c, 0)["mixer"].update(dim=300, rot={"dims": 8, "base": 10.0})), 6, "256")
    bad = folder(tmp_path, good, tensors, "r")
    os.unlink(os.path.join(bad, "model.safetensors"))
    refused(bad, 7)


# ---- the plain implementation against other forms of its equations --------------------------------------------------------------------------
def test_rotation_keeps_lengths_and_depends_on_distances():
    r = np.random.default_rng(0)
    a, b = r.normal(size=(1, 1, 12)), r.normal(size=(1, 1, 12))
    at = lambda x, p: plain.rotate(x, [p], 8, 100.0)[0, 0]
    for p, s in ((0, 5), (3, 8), (1000, 1005)):
        assert np.linalg.norm(at(a, p)) == pytest.approx(np.linalg.norm(a))
        assert at(a, p) @ at(b, s) == pytest.approx(at(a, 0) @ at(b, 5))
    np.testing.assert_array_equal(at(a, 7)[8:], a[0, 0, 8:])
    z = (a[0, 0, :4] + 1j * a[0, 0, 4:8]) * np.exp(1j * 7 * 100.0 ** (-np.arange(4) / 4))  # pair (i, i + 4) as a complex number
    np.testing.assert_allclose(at(a, 7)[:8], np.concatenate([z.real, z.imag]), atol=1e-12)


def test_retention_is_its_sum_over_the_past():
    r = np.random.default_rng(1)
    qs, ks, vs = r.normal(size=(9, 5)), r.normal(size=(9, 5)), r.normal(size=(9, 3))
    got = plain.retention_state(qs, ks, vs, 0.8)
    for t in range(9):
        np.testing.assert_allclose(got[t], sum(0.8 ** (t - s) * (qs[t] @ ks[s]) * vs[s] for s in range(t + 1)), atol=1e-12)


def test_attention_written_out():
    r = np.random.default_rng(2)
    c = {"heads": 4, "kv_heads": 2, "dim": 3, "vdim": 5, "scale": 0.7, "q_temp": {"coef": 0.5, "every": 4}}
    w = {"q": r.normal(size=(12, 6)), "k": r.normal(size=(6, 6)), "v": r.normal(size=(10, 6)), "q.norm": r.uniform(0.5, 1.5, 12), "k.norm": r.uniform(0.5, 1.5, 6), "pb": r.normal(size=4), "o": np.eye(20)}
    h = r.normal(size=(11, 6))
    got = plain.sigmoid_attention(h, w, c, 1e-5).reshape(11, 4, 5)
    for i in (0, 2, 3, 4, 10):
        for a in range(4):
            want = np.zeros(5)
            qq = w["q"] @ h[i]
            qq = (qq / np.sqrt((qq ** 2).mean() + 1e-5) * w["q.norm"])[3 * a:3 * a + 3] * (1 + 0.5 * np.log((i + 1) // 4 + 1))
            for j in range(i + 1):
                k, v = w["k"] @ h[j], (w["v"] @ h[j])[5 * (a // 2):5 * (a // 2) + 5]
                k = (k / np.sqrt((k ** 2).mean() + 1e-5) * w["k.norm"])[3 * (a // 2):3 * (a // 2) + 3]
                score = 0.7 * (qq @ k) - (i - j) * 2.0 ** (-2 * (a + 1)) + w["pb"][a]
                want += v / np.sqrt((v ** 2).mean() + 1e-5) / (1 + np.exp(-score))
            np.testing.assert_allclose(got[i, a], want, atol=1e-10)


def test_the_groups_of_the_router():
    c = {"experts": 6, "top": 2, "scale": 2.0, "groups": {"count": 3, "keep": 1}}
    z = np.array([1.0, 0.9, 1.2, -5.0, 1.1, 1.15])
    s = np.exp(z) / np.exp(z).sum()
    chosen, weights = plain.route(z, c)  # the best group is the second, although its other expert is the worst of all
    assert chosen.tolist() == [2, 3]
    np.testing.assert_allclose(weights, 2.0 * s[[2, 3]])
    c["groups"]["keep"] = 2
    assert plain.route(z, c)[0].tolist() == [2, 5]
    c["groups"]["keep"] = 3
    assert plain.route(np.array([1.3, 0.9, 1.2, -5.0, 1.1, 1.15]), c)[0].tolist() == [0, 2]


def test_depth_averages_of_unit_vectors_pass_the_stream_on():
    cfg = config()
    w = {k: mf.bf16_floats(v).astype(np.float64) for k, v in mf.random_tosevik(cfg, 3).items()}
    ids = np.arange(12) % 19
    for i in range(3):
        w[f"l{i}.dwa"] = np.eye(i + 2)[0]  # only the embedding output
    stream, logits = plain.tosevik_stream(cfg, w, ids)
    x0 = plain.dynamic_tanh(w["embed"][ids], w["embed.norm"], w["embed.norm.b"], w["embed.norm.alpha"])
    for s in stream:
        np.testing.assert_allclose(s, x0)
    np.testing.assert_allclose(logits, plain.dynamic_tanh(x0, w["final.norm"], w["final.norm.b"], w["final.norm.alpha"]) @ w["head"].T)


def test_no_position_depends_on_later_tokens():
    cfg = config()
    w = {k: mf.bf16_floats(v).astype(np.float64) for k, v in mf.random_tosevik(cfg, 3).items()}
    ids = np.random.default_rng(2).integers(0, 19, 31)
    np.testing.assert_allclose(plain.tosevik(cfg, w, ids)[:19], plain.tosevik(cfg, w, ids[:19]), atol=1e-9)
