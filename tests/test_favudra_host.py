"""Favudra design on the host: config reader and writer, refusals, merged layouts and packing, a checkpoint whose bottleneck
rank only the tensors know, and the restatement's own sanity (causality, convolution, window, bias, sink, cap, recurrence)."""
import copy
import math

import pytest
import torch

import favudra_oracle as fo
from tinygpt_b200 import loader, models


def doc():
    attn = {"heads": 6, "kv_heads": 2, "dim": 10, "vdim": 14, "conv": 4, "scale": 0.3, "softcap": 7.0, "rot": {"base": 90.0, "dims": 6}}
    return {"architecture": "Favudra", "embedding": {"scale": 2.5}, "logit_scale": 0.4, "norm": {"eps": 1e-5}, "vocab": 40, "width": 24,
            "layers": [
                {"type": "attention", "mixer": dict(attn), "mlp": {"kind": "dense", "ff": 20}},
                {"type": "gla", "mixer": {"heads": 2, "dim": 6, "vdim": 9, "tau": 5.0}, "mlp": None},
                {"type": "attention", "mixer": dict(attn, heads=2, softcap=3.0, kv_from=0), "mlp": None},
                {"type": "attention_2", "mixer": {"heads": 3, "kv_heads": 1, "dim": 7, "vdim": 7, "scale": 0.2, "mask": {"size": 5}},
                 "mlp": {"kind": "dense", "ff": 12}}]}


SHAPES = {"l1.mix.a1": (3, 24)}


def spec():
    return models.favudra_from_config(doc(), shapes=SHAPES)


def weights(s, seed=0):
    w = models.synth_favudra_weights(s, seed)
    return w, {k: v.double() for k, v in w.items()}


def test_registry_and_config_round_trip():
    assert "Favudra" in models.ARCHITECTURES and models.ARCHITECTURES["Favudra"].with_shapes
    s = models.ARCHITECTURES["Favudra"](doc(), SHAPES)
    assert models.favudra_config(s) == doc()
    a, g, q, t = s.layers
    assert a.prep.conv == 4 and a.prep.head_norm and a.prep.rot_interleaved and a.attn.sink and a.attn.softcap == 7.0 and a.attn.window == 0
    assert g.gla == models.GlaSpec(2, 6, 9, 5.0, 3) and g.ff == 0
    assert q.kv_from == 0 and q.attn.softcap == 3.0
    assert t.attn.values_are_keys and t.attn.distance_bias and not t.attn.sink and t.attn.window == 5 and t.prep is None
    assert s.block == "sandwich" and s.norm_kind == "rms" and s.embed_scale == 2.5 and s.logit_scale == 0.4


@pytest.mark.parametrize("change", ["type", "mlp", "heads", "rot", "kv_later", "kv_tied", "kv_chain", "kv_sizes", "vdim", "rank", "tau"])
def test_refused_configs(change):
    d, shapes = doc(), dict(SHAPES)
    L = d["layers"]
    if change == "type":
        L[1]["type"] = "delta"
    elif change == "mlp":
        L[0]["mlp"]["kind"] = "moe"
    elif change == "heads":
        L[0]["mixer"]["heads"] = 5
    elif change == "rot":
        L[0]["mixer"]["rot"]["dims"] = 12
    elif change == "kv_later":
        L[2]["mixer"]["kv_from"] = 2
    elif change == "kv_tied":
        L.append(copy.deepcopy(L[2]))
        L[4]["mixer"]["kv_from"] = 3
    elif change == "kv_chain":
        L.append(copy.deepcopy(L[2]))
        L[4]["mixer"]["kv_from"] = 2
    elif change == "kv_sizes":
        L[2]["mixer"]["vdim"] = 13
    elif change == "vdim":
        L[3]["mixer"]["vdim"] = 8
    elif change == "rank":
        shapes = {}
    elif change == "tau":
        L[1]["mixer"]["tau"] = 0
    with pytest.raises(ValueError):
        models.favudra_from_config(d, shapes=shapes)


def test_optional_entries_may_be_absent():
    d = doc()
    del d["layers"][0]["mixer"]["rot"], d["layers"][2]["mixer"]["rot"], d["layers"][0]["mixer"]["softcap"], d["layers"][3]["mixer"]["mask"]
    s = models.favudra_from_config(d, shapes=SHAPES)
    assert s.layers[0].prep.rot is None and s.layers[0].attn.softcap == 0.0 and s.layers[3].attn.window == 0


def test_slopes():
    a = models.AttnSpec(heads=3, kv_heads=1, dim=4, vdim=4, scale=1.0)
    assert a.slopes().tolist() == pytest.approx([2 ** (-8 / 3), 2 ** (-16 / 3), 2 ** -8]) == fo.slopes(3)


def test_layout_and_packing():
    s = spec()
    w, _ = weights(s)
    p = models.pack_weights(s, w, device="cpu", dtype=torch.float32)
    lay = s.mix_layout(0)
    assert (lay.off_q, lay.off_k, lay.off_v, lay.n_in, lay.k_out) == (0, 64, 88, 120, 84)
    assert torch.equal(p["l0.w_in"][64:84], w["l0.mix.k"].float()) and not p["l0.w_in"][84:88].any()
    taps = p["l0.conv_w"].view(4, 120)
    assert torch.equal(taps[:, 88:116], w["l0.mix.v.conv"].float().t()) and torch.equal(taps[3, :60], w["l0.mix.q.conv"][:, 3].float())
    lay = s.mix_layout(1)
    assert (lay.off_k, lay.off_v, lay.off_g, lay.off_up, lay.n_in) == (16, 32, 56, 80, 88)
    assert torch.equal(p["l1.w_in"][80:83], w["l1.mix.a1"].float()) and p["l1.a2"].shape == (12, 8) and not p["l1.a2"][:, 3:].any()
    assert s.mix_layout(2).n_in == 24 and "l2.k_norm" not in p
    lay = s.mix_layout(3)
    assert lay.off_v == lay.off_k == 24 and lay.n_in == 32 and p["l3.slopes"].tolist() == pytest.approx(fo.slopes(3))
    assert torch.equal(p["l0.post_norm"], 1 + w["l0.norm1b"].float())
    assert torch.allclose(p["final_norm"], (1 + w["final.norm"].float()) * 0.4)
    assert torch.equal(p["l0.w_ff_in"], torch.cat([w["l0.mlp.gate"], w["l0.mlp.up"]]).float())
    n = 24 * (60 + 20 + 28 + 84 + 3 * 20) + 24 * (24 + 54 + 3) + 12 * 3 + 24 * (20 + 28) + 24 * (21 + 7 + 21 + 36) + 40 * 24
    assert s.weight_params() == n


def test_checkpoint_round_trip_finds_the_rank_in_the_tensors(tmp_path):
    s = spec()
    w, _ = weights(s)
    models.save_stack_checkpoint(s, w, tmp_path)
    s2, p2 = loader.load_model(tmp_path, device="cpu", dtype=torch.float32, max_ctx=64, max_slots=2)
    assert s2.layers == s.layers and s2.max_ctx == 64
    p = models.pack_weights(s, w, device="cpu", dtype=torch.float32)
    assert p.keys() == p2.keys() and all(torch.equal(p[k], p2[k]) for k in p)
    (tmp_path / "model.safetensors").write_bytes((tmp_path / "model.safetensors").read_bytes().replace(b"l1.mix.a2.b", b"l1.mix.a2.x"))
    with pytest.raises(loader.LoaderError):
        loader.load_model(tmp_path, device="cpu", dtype=torch.float32)


# ------------------------------------------------------------------------------------------- the restatement itself
def toks(n, seed=1):
    return torch.randint(0, 40, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def test_restatement_is_causal_and_independent_of_cuts():
    d = doc()
    _, w = weights(spec())
    t = toks(25)
    whole = fo.forward(d, w, t)
    seq = fo.Sequence(d)
    parts = torch.cat([fo.forward(d, w, t[a:b], seq) for a, b in ((0, 1), (1, 3), (3, 14), (14, 15), (15, 25))])
    assert torch.allclose(whole, parts, atol=1e-9)
    other = list(t)
    other[20] = (t[20] + 1) % 40
    z = fo.forward(d, w, other)
    assert torch.allclose(z[:20], whole[:20], atol=1e-12) and not torch.allclose(z[20:], whole[20:], atol=1e-3)


def test_restatement_convolution_and_rotation():
    x = torch.arange(1.0, 7.0, dtype=torch.float64).view(6, 1)
    y, last = fo.short_conv(x, torch.tensor([[100.0, 10.0, 1.0]], dtype=torch.float64), None)
    assert y[:, 0].tolist() == [1, 12, 123, 234, 345, 456] and last[:, 0].tolist() == [5, 6]
    y2, _ = fo.short_conv(x[:1] + 6, torch.tensor([[100.0, 10.0, 1.0]], dtype=torch.float64), last)
    assert y2.item() == 567
    v = torch.tensor([[[1.0, 0.0, 1.0, 0.0, 5.0]]], dtype=torch.float64)
    r = fo.rotate_pairs(v, torch.tensor([3]), {"base": 16.0, "dims": 4})[0, 0]
    assert r.tolist() == pytest.approx([math.cos(3), math.sin(3), math.cos(0.75), math.sin(0.75), 5.0])


def test_restatement_sink_cap_window_and_bias():
    vis = torch.tensor([[True, True, False]])
    s = torch.tensor([[1.0, -2.0, 9.0]], dtype=torch.float64)
    e = [math.exp(1), math.exp(-2)]
    assert fo.softmax_weights(s, vis, True)[0].tolist() == pytest.approx([e[0] / (1 + sum(e)), e[1] / (1 + sum(e)), 0.0])
    assert fo.softmax_weights(s, vis, False)[0].tolist() == pytest.approx([e[0] / sum(e), e[1] / sum(e), 0.0])
    assert fo.capped(torch.tensor(300.0), 5.0) == pytest.approx(5.0) and fo.capped(torch.tensor(3.0), 0.0) == 3.0
    # equal keys: the weights follow the bias alone, over the window's positions
    m = {"heads": 2, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 1.0, "mask": {"size": 3}}
    w = {"mix.q": torch.zeros(2, 1, dtype=torch.float64), "mix.o": torch.eye(2, dtype=torch.float64)}
    keys = torch.tensor([[[100.0]], [[1.0]], [[0.0]], [[0.0]]], dtype=torch.float64)
    out = fo.biased_attention(torch.ones(1, 1, dtype=torch.float64), torch.tensor([3]), m, w, "", keys, torch.arange(4))
    for h, sl in enumerate((2.0 ** -4, 2.0 ** -8)):
        e = [math.exp(-sl * k) for k in range(3)]
        assert out[0, h].item() == pytest.approx(e[2] / sum(e))


def test_restatement_recurrence_closed_form():
    """After one token o = (k·q) v; after two the first is decayed per key channel."""
    g = torch.Generator().manual_seed(3)
    H, dk, dv, W = 1, 3, 2, 4
    w = {n: torch.randn(s, generator=g, dtype=torch.float64) for n, s in
         {"mix.q": (dk, W), "mix.k": (dk, W), "mix.v": (dv, W), "mix.g": (dv, W), "mix.o": (dv, dv), "mix.a1": (2, W), "mix.a2": (dk, 2),
          "mix.a2.b": (dk,)}.items()}
    w["mix.norm"] = torch.ones(dv, dtype=torch.float64)
    h = torch.randn(2, W, generator=g, dtype=torch.float64)
    m = {"heads": H, "dim": dk, "vdim": dv, "tau": 2.0}
    got, S = fo.gla_mixer(h, m, w, "", 0.0, None)
    q, k, v = h @ w["mix.q"].T / math.sqrt(dk), h @ w["mix.k"].T, h @ w["mix.v"].T
    alpha = torch.sigmoid(h @ w["mix.a1"].T @ w["mix.a2"].T + w["mix.a2.b"]) ** 0.5
    want = torch.stack([(k[0] @ q[0]) * v[0], ((alpha[1] * k[0]) @ q[1]) * v[0] + (k[1] @ q[1]) * v[1]])
    want = want / want.pow(2).mean(-1, keepdim=True).sqrt()
    z = h @ w["mix.g"].T
    assert torch.allclose(got, (want * z * torch.sigmoid(z)) @ w["mix.o"].T)
    assert torch.allclose(S[0], alpha[1][:, None] * torch.outer(k[0], v[0]) + torch.outer(k[1], v[1]))
