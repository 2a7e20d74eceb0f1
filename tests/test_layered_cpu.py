"""Layered models without a GPU: the folder reader behind ``quintrit_b200_gguf_describe`` (config.json, safetensors, what it refuses), and the plain
implementation against other ways of writing the same equations."""
import json
import os
import struct

import numpy as np
import pytest

import quintrit_b200 as q
from oracle import layered as plain
from quintrit_b200 import model_folder as mf

LAYERS = [mf.mamba2(4, 8, 12, groups=2, conv=3, norm_groups=2, ff=24), mf.attention(4, 2, 8, 12, 9, 4, scale=0.25), mf.hgrn2(2, 8, 16, ff=20)]


def folder(tmp_path, config=None, tensors=None, name="m"):
    config = config or mf.lasosun_config(LAYERS, 20, 17, 50, eps=2e-5, embed_scale=2.5)
    return mf.write_folder(str(tmp_path / name), config, tensors if tensors is not None else mf.random_lasosun(config, 1))


def test_describe_reads_every_size_and_constant(tmp_path):
    d = q.gguf_describe(folder(tmp_path))
    assert (d["architecture"], d["vocab_size"], d["hidden_size"], d["num_layers"], d["context_length"], d["tied"]) == ("Lasosun", "17", "20", "3", "50", "1")
    assert float(d["rms_norm_eps"]) == pytest.approx(2e-5) and float(d["embed_scale"]) == 2.5
    assert d["layer_0"] == "mamba2 heads=4 vdim=8 state=12 groups=2 conv=3 norm_groups=2 ff=24"
    assert d["layer_1"].startswith("attention heads=4 vdim=12 dim=8 kv_heads=2 window=9 pool=4 scale=0.25") and d["layer_1"].endswith("ff=0")
    assert d["layer_2"] == "hgrn2 heads=2 vdim=16 dim=8 ff=20"
    shapes = {t["name"]: t["shape"] for t in d["tensors"]}
    assert shapes == {k: tuple(v) for k, v in mf.lasosun_shapes(mf.lasosun_config(LAYERS, 20, 17, 50)).items()}
    assert all(t["type"] == "BF16" for t in d["tensors"])


def refused(path, code, text=""):
    with pytest.raises(q.QuintritError) as e:
        q.gguf_describe(path)
    assert e.value.code == code and text in str(e.value), str(e.value)


def test_config_mistakes_are_named(tmp_path):
    good = mf.lasosun_config(LAYERS, 20, 17, 50)
    tensors = mf.random_lasosun(good, 1)

    def variant(name, change):
        c = json.loads(json.dumps(good))
        change(c)
        return folder(tmp_path, c, tensors, name)

    refused(variant("a", lambda c: c.update(architecture="Other")), 6, "Other")
    refused(variant("b", lambda c: c.pop("width")), 10, "width")
    refused(variant("c", lambda c: c["layers"][0]["mixer"].pop("state")), 10, "layers[0].mixer.state")
    refused(variant("d", lambda c: c["layers"][1]["mixer"]["mask"].update(size=-3)), 10, "mask.size")
    refused(variant("e", lambda c: c["layers"][2].update(type="rwkv")), 10, "rwkv")
    refused(variant("f", lambda c: c["layers"][0]["mlp"].update(kind="moe")), 10, "moe")
    refused(variant("g", lambda c: c["layers"][0]["mixer"].update(groups=3)), 6, "groups")
    refused(variant("h", lambda c: c["layers"][1]["mixer"].update(kv_heads=3)), 6, "kv_heads")
    refused(variant("i", lambda c: c["layers"][0]["mixer"].update(norm_groups=5)), 6, "norm_groups")
    refused(variant("j", lambda c: c.update(norm={"eps": "small"})), 10, "norm.eps")
    empty = tmp_path / "nothing"
    empty.mkdir()
    refused(str(empty), 7)
    bad = variant("k", lambda c: None)
    for text in ("{", '{"a": [1, 2,]}', '{"a" 1}', "[1]", '{"a": 1} x', '{"a": tru}', '{"a": "\\q"}'):
        open(os.path.join(bad, "config.json"), "w").write(text)
        refused(bad, 8)


def test_json_text_is_read_whole(tmp_path):
    path = folder(tmp_path)
    c = json.load(open(os.path.join(path, "config.json")))
    c["note"] = 'quoted "text", \\ and é \U0001f600'
    c["norm"]["eps"] = 3e-7
    c["width"] = 2.0e1
    json.dump(c, open(os.path.join(path, "config.json"), "w"), indent=1)
    d = q.gguf_describe(path)
    assert d["hidden_size"] == "20" and float(d["rms_norm_eps"]) == pytest.approx(3e-7)


def test_safetensors_mistakes(tmp_path):
    path = folder(tmp_path)
    file = os.path.join(path, "model.safetensors")
    raw = open(file, "rb").read()
    n = struct.unpack("<Q", raw[:8])[0]
    for broken in (b"", raw[:4], struct.pack("<Q", 1 << 60) + raw[8:], raw[:8] + b"x" * n + raw[8 + n:], raw[:-3]):
        open(file, "wb").write(broken)
        refused(path, 8)
    os.unlink(file)
    refused(path, 7)


def test_without_a_device_nothing_is_computed(tmp_path):
    if q.device_count() > 0:
        pytest.skip("a GPU is present")
    with pytest.raises(q.QuintritError) as e:
        q.Decoder.open(folder(tmp_path))
    assert e.value.code == 15


# ---- the plain implementation against other forms of its equations --------------------------------------------------------------------------
def rng_weights(config, seed):
    return {k: mf.bf16_floats(v).astype(np.float64) for k, v in mf.random_lasosun(config, seed).items()}


def test_short_convolution_is_a_correlation():
    r = np.random.default_rng(0)
    u, w, b = r.normal(size=(11, 3)), r.normal(size=(3, 4)), r.normal(size=3)
    got = plain.short_conv(u, w, b)
    for c in range(3):
        np.testing.assert_allclose(got[:, c], np.convolve(u[:, c], w[c, ::-1])[:11] + b[c], atol=1e-12)


def test_recurrences_equal_their_sums_over_the_past():
    """S_t written out: every earlier token, times the decays since."""
    r = np.random.default_rng(1)
    c = {"heads": 2, "dim": 5, "vdim": 4}
    w = {"q": r.normal(size=(10, 6)), "f": r.normal(size=(10, 6)), "v": r.normal(size=(8, 6)), "f.b": r.normal(size=10), "lower": r.uniform(0, 0.9, 10), "norm": np.ones(4), "o": np.eye(8)}
    h = r.normal(size=(9, 6))
    q_, v = plain.silu(h @ w["q"].T), h @ w["v"].T
    f = w["lower"] + (1 - w["lower"]) * plain.sigmoid(h @ w["f"].T + w["f.b"])
    want = np.zeros((9, 8))
    for t in range(9):
        for s in range(t + 1):
            k = (1 - f[s]) * np.prod(f[s + 1:t + 1], axis=0) * q_[t]
            want[t] += np.repeat(k.reshape(2, 5).sum(1), 4) * v[s]
    want = plain.rms_norm(want.reshape(9, 2, 4), 1.0, 1e-6).reshape(9, 8)
    np.testing.assert_allclose(plain.hgrn2(h, w, c, 1e-6), want, atol=1e-10)

    c = {"heads": 2, "vdim": 4, "state": 3, "groups": 1, "conv": 1, "norm_groups": 1}
    w = {"in": r.normal(size=(8 + 8 + 6 + 2, 6)), "conv": np.ones((14, 1)), "conv.b": np.zeros(14), "dt_bias": r.normal(size=2), "A_log": r.normal(size=2), "D": r.normal(size=2), "norm": np.ones(8), "o": np.eye(8)}
    p = h @ w["in"].T
    x, B, C, dt = plain.silu(p[:, 8:16]), plain.silu(p[:, 16:19]), plain.silu(p[:, 19:22]), np.log1p(np.exp(p[:, 22:] + w["dt_bias"]))
    y = np.zeros((9, 2, 4))
    for t in range(9):
        for k in range(2):
            for s in range(t + 1):
                y[t, k] += np.exp(-np.exp(w["A_log"][k]) * dt[s + 1:t + 1, k].sum()) * dt[s, k] * (B[s] @ C[t]) * x[s, 4 * k:4 * k + 4]
            y[t, k] += w["D"][k] * x[t, 4 * k:4 * k + 4]
    np.testing.assert_allclose(plain.mamba2(h, w, c, 1e-6), plain.rms_norm(y.reshape(9, 8) * plain.silu(p[:, :8]), 1.0, 1e-6), atol=1e-10)


def test_what_a_position_sees():
    assert plain.visible(0, 4, 3) == ([0], [])
    assert plain.visible(5, 4, 3) == ([2, 3, 4, 5], [])        # block 0 ends at 2, which is still in the window
    assert plain.visible(6, 4, 3) == ([3, 4, 5, 6], [0])
    assert plain.visible(8, 4, 3) == ([5, 6, 7, 8], [0])       # 3 and 4 have left, their block has not
    assert plain.visible(9, 4, 3) == ([6, 7, 8, 9], [0, 1])
    for i in range(40):  # every position once or not at all, never a part of a block twice
        tokens, blocks = plain.visible(i, 7, 4)
        inside = [j for b in blocks for j in range(4 * b, 4 * b + 4)]
        assert not set(tokens) & set(inside) and len(inside) == len(set(inside)) and max(inside, default=i - 7) <= i - 7


def test_no_position_depends_on_later_tokens():
    config = mf.lasosun_config(LAYERS, 20, 17, 50)
    w = rng_weights(config, 3)
    ids = np.random.default_rng(2).integers(0, 17, 31)
    a, b = plain.lasosun(config, w, ids), plain.lasosun(config, w, ids[:19])
    np.testing.assert_allclose(a[:19], b, atol=1e-9)
