"""Vazatar without a GPU: configuration, layout, checkpoint boundary, step tables, oracle sanity."""
import json
import math

import numpy as np
import pytest
import torch

import vazatar_oracle as O
import vazatar_util as U
from async_grpo_nccl_b200 import checkpoint as ckpt
from async_grpo_nccl_b200.models.listed import host_batch, split_batch
from async_grpo_nccl_b200.models.registry import PRESETS, architecture_of, config_from_dict, make_layout, require_trainable, resolve_model_config


def test_registry_chooses_by_config(tmp_path):
    cfg = resolve_model_config(U.save_checkpoint(tmp_path / "m", "odd"))
    assert architecture_of(cfg).name == "Vazatar" and cfg.layers[0].mixer.chunk == 48 and cfg.layers[1].mixer.state == 5
    assert cfg.runs() == [(0, False), (1, True), (2, False), (1, True), (2, False)]
    with pytest.raises(NotImplementedError):
        require_trainable(cfg)
    assert config_from_dict({"preset": "vazatar-tiny"}) == PRESETS["vazatar-tiny"]
    assert PRESETS["vazatar-1.5b"].first_layers(8).runs()[-1][0] == 7


@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_config_round_trip(name):
    cfg = config_from_dict(U.CONFIGS[name])
    assert config_from_dict(json.loads(json.dumps(cfg.to_hf_dict()))) == cfg
    assert cfg.num_parameters() == sum(v.numel() for v in U.weights(name).values())
    assert cfg.runs() == O.layer_order(U.CONFIGS[name])


def test_bad_configs_are_refused():
    def changed(layer, where, **kw):
        c = json.loads(json.dumps(U.CONFIGS["odd"]))
        d = c["layers"][layer]
        for k in where:
            d = d[k]
        d.update(kw)
        return c

    bad = [changed(0, ["mixer"], kv_heads=4), changed(0, ["mixer", "mask"], size=0), changed(0, ["mixer", "rot"], dims=7),
           changed(0, ["mixer", "rot"], dims=42), changed(1, ["mixer"], state=0), changed(1, [], type="mamba9"), changed(0, ["mlp"], kind="moe")]
    loop = json.loads(json.dumps(U.CONFIGS["odd"]))
    loop["loop"]["stop"] = 4
    for c in bad + [loop]:
        with pytest.raises(ValueError):
            config_from_dict(c)


@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_checkpoint_loads_and_saves(tmp_path, name):
    cfg = resolve_model_config(U.save_checkpoint(tmp_path / "a", name))
    layout = make_layout(cfg)
    flat = ckpt.load_hf_model(str(tmp_path / "a"), layout)
    assert int((flat != 0).sum()) <= cfg.num_parameters()  # padding stays zero
    ckpt.save_hf_model(str(tmp_path / "b"), cfg, layout, flat)
    from safetensors.torch import load_file

    saved, want = load_file(str(tmp_path / "b" / "model.safetensors")), U.weights(name)
    assert set(saved) == set(want)
    for k, v in want.items():
        assert saved[k].shape == v.shape and torch.equal(saved[k].double(), v), k
    assert torch.equal(ckpt.load_hf_model(str(tmp_path / "b"), layout), flat)


def test_checkpoint_errors(tmp_path):
    from safetensors.torch import save_file

    layout = make_layout(config_from_dict(U.CONFIGS["odd"]))
    w = {k: v.to(torch.bfloat16).contiguous() for k, v in U.weights("odd").items()}
    for breakage in ("missing", "shape", "extra"):
        p = tmp_path / breakage
        p.mkdir()
        x = dict(w)
        if breakage == "missing":
            del x["l1.mix.dt.b"]
        elif breakage == "shape":
            x["loop.in"] = x["loop.in"][:, :-1].contiguous()
        else:
            x["l2.mlp.up"] = torch.zeros(3, 3, dtype=torch.bfloat16)  # that layer has no feed-forward
        save_file(x, str(p / "model.safetensors"))
        with pytest.raises((KeyError, ValueError)):
            ckpt.load_hf_model(str(p), layout)
    # the norm ahead of an absent feed-forward may be there and is not read
    d = U.save_checkpoint(tmp_path / "unused", "odd", **{"l2.norm2": torch.ones(100, dtype=torch.float64)})
    assert torch.equal(ckpt.load_hf_model(d, layout), ckpt.load_hf_model(U.save_checkpoint(tmp_path / "without", "odd"), layout))


def test_random_init_clears_padding():
    cfg = PRESETS["vazatar-tiny"]
    layout = make_layout(cfg)
    flat, dev = torch.empty(layout.total), torch.empty(layout.total)
    layout.init_random_(flat, 3)
    layout.init_random_device_(dev, 3)
    for f in (flat, dev):
        assert 0 < int((f != 0).sum()) <= cfg.num_parameters()
        a = layout.view(f, "layers.1.A_log")
        assert torch.allclose(a[0], torch.log(torch.arange(1, 9).float())) and float(layout.view(f, "layers.1.conv")[:, -1].mean()) > 0.9


@pytest.mark.parametrize("name", ["odd", "chunks", "plain"])
def test_frequencies(name):
    for spec, l in zip(config_from_dict(U.CONFIGS[name]).layers, U.CONFIGS[name]["layers"]):
        if l["type"] == "attention":
            r = l["mixer"]["rot"]
            assert np.allclose(spec.mixer.rot.frequencies(), O.frequencies(r["dims"], r["base"], r["scaling"]), rtol=1e-14)
    r = config_from_dict(U.CONFIGS["odd"]).layers[0].mixer.rot  # wavelengths below 18, between, above 90
    f, plain = r.frequencies(), [500.0 ** (-2 * i / 32) for i in range(16)]
    kinds = {"kept" if a == b else "slowed" if math.isclose(a, b / 3) else "between" for a, b in zip(f, plain)}
    assert kinds == {"kept", "slowed", "between"}


def test_step_tables():
    flat, where = host_batch([(3, 5, np.arange(130)), (1, 0, np.asarray([7, 8])), (2, 100, np.arange(3))], [4], 1, [48, 33])
    _, sb = split_batch(torch.from_numpy(flat), where, torch.zeros(4, 4, dtype=torch.int32))
    assert sb.segs.tolist() == [[0, 130, 3, 5], [130, 2, 1, 0], [132, 3, 2, 100]] and sb.segs.storage_offset() % 4 == 0
    # token 100 lies in the chunks that start at 96 and 99: pages from 96 on
    assert sb.pages.tolist() == [[3, p] for p in range(9)] + [[1, 0], [2, 6]]
    assert sorted(map(tuple, sb.tiles.tolist())) == [(0, 128, 5, 0), (128, 2, 133, 0), (130, 2, 0, 144), (132, 3, 100, 160 - 96)]
    assert sb.ring_rows[4].tolist() == [126, 127, 128, 129, 130, 131, 132, 133, 134]


# ---- the oracle's own mechanisms on cases that can be worked out by hand ----
def test_oracle_mechanisms():
    d = dict(dtype=torch.float64)
    x = torch.tensor([[3.0, 4.0]], **d)
    assert torch.allclose(O.norm_zero_centred(x, torch.tensor([0.0, 1.0], **d), 0.0), x / math.sqrt(12.5) * torch.tensor([1.0, 2.0], **d))
    u = torch.tensor([[1.0], [10.0], [100.0]], **d)
    assert O.causal_conv(u, torch.tensor([[2.0, 3.0]], **d), torch.tensor([5.0], **d)).flatten().tolist() == [8.0, 37.0, 325.0]
    assert torch.allclose(O.softplus(torch.tensor([0.0, 40.0, -40.0], **d)), torch.tensor([math.log(2), 40.0, math.exp(-40)], **d))
    assert O.chunk_mask(5, 2).int().tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [0, 0, 1, 0, 0], [0, 0, 1, 1, 0], [0, 0, 0, 0, 1]]
    q = torch.tensor([[[1.0, 0.0, 7.0]], [[1.0, 0.0, 7.0]]], **d)
    assert torch.allclose(O.rotate(q, [0.5])[1, 0], torch.tensor([math.cos(0.5), math.sin(0.5), 7.0], **d))
    one = torch.ones(2, 1, **d)
    y, S = O.selective_scan(one, one * math.log(2), -one[:1], one, one, torch.tensor([10.0], **d))
    ln2 = math.log(2)
    assert torch.allclose(y.flatten(), torch.tensor([ln2 + 10, 1.5 * ln2 + 10], **d)) and float(S) == pytest.approx(1.5 * ln2)
    half = O.selective_scan(one[:1], one[:1] * ln2, -one[:1], one[:1], one[:1], torch.tensor([10.0], **d))[1]
    assert torch.allclose(O.selective_scan(one[1:], one[1:] * ln2, -one[:1], one[1:], one[1:], torch.tensor([10.0], **d), half)[1], S)


def test_a_planted_mistake_shows_in_the_oracle():
    """Each mechanism left out (or off by one) changes the oracle's logits by far more than the tests' tolerances."""
    name, n = "odd", 60
    base, cfg, w, t = U.oracle_logits(name, n), U.CONFIGS[name], U.weights(name), U.tokens(name, n)

    def changed(edit_cfg=None, edit_w=None):
        c, x = json.loads(json.dumps(cfg)), dict(w)
        if edit_cfg:
            edit_cfg(c)
        if edit_w:
            x = {k: edit_w(k, v) for k, v in x.items()}
        return U.worst_row(O.forward(c, x, t), base)

    def attention(**kw):
        def edit(c):
            for l in c["layers"]:
                if l["type"] == "attention":
                    l["mixer"].update({k: v(l["mixer"][k]) for k, v in kw.items()})
        return edit

    assert changed(attention(mask=lambda m: {"size": m["size"] + 1})) > 0.1
    assert changed(attention(softcap=lambda c: 1e9)) > 1e-3
    assert changed(attention(rot=lambda r: {**r, "dims": r["dims"] - 2})) > 0.1
    assert changed(attention(rot=lambda r: {**r, "scaling": {**r["scaling"], "factor": 1.0}})) > 0.05
    assert changed(lambda c: c["loop"].update(times=1)) > 0.1
    assert changed(lambda c: c.update(logit_softcap=1e9)) > 0.1
    assert changed(edit_w=lambda k, v: v * 0 + 1 if k.endswith("k.norm") else v) > 0.1
    assert changed(edit_w=lambda k, v: v * torch.tensor([0.0, 1, 1]) if k.endswith("mix.conv") else v) > 0.05
    for leaf in ("conv.b", "dt.b", "mix.D", "norm2"):
        assert changed(edit_w=lambda k, v: v * 0 if k.endswith(leaf) else v) > 0.05
    assert changed(edit_w=lambda k, v: torch.cat([v[:, :100], v[:, 100:] * 0], 1) if k == "loop.in" else v) > 0.1
