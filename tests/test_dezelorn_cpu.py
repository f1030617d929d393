"""Dezelorn without a GPU: configuration, layout, checkpoint boundary, step tables, scheduler additions, oracle sanity."""
import json

import numpy as np
import pytest
import torch

import dezelorn_oracle as O
import dezelorn_util as U
from async_grpo_nccl_b200 import checkpoint as ckpt
from async_grpo_nccl_b200.models.config import ModelConfig
from async_grpo_nccl_b200.models.listed import host_batch, split_batch
from async_grpo_nccl_b200.models.registry import PRESETS, architecture_of, config_from_dict, make_layout, require_trainable, resolve_model_config


def test_registry_chooses_by_config(tmp_path):
    d = U.save_checkpoint(tmp_path / "m", "odd")
    cfg = resolve_model_config(d)
    assert architecture_of(cfg).name == "Dezelorn" and cfg.vocab_size == 333 and cfg.layers[0].mixer.window == 48
    assert isinstance(resolve_model_config("tiny"), ModelConfig)
    assert architecture_of(resolve_model_config("qwen2.5-1.5b")).trainable
    with pytest.raises(NotImplementedError):
        require_trainable(cfg)
    with pytest.raises(ValueError):
        config_from_dict({**U.CONFIGS["odd"], "architecture": "Unheard"})


@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_config_round_trip(name):
    cfg = config_from_dict(U.CONFIGS[name])
    again = config_from_dict(json.loads(json.dumps(cfg.to_hf_dict())))
    assert again == cfg
    assert cfg.num_parameters() == sum(v.numel() for v in U.weights(name).values())


def test_bad_configs_are_refused():
    base = U.CONFIGS["odd"]

    def with_mixer(**kw):
        c = json.loads(json.dumps(base))
        c["layers"][1]["mixer"].update(kw)
        return c

    for bad in (with_mixer(kv_heads=4), with_mixer(vdim=41), with_mixer(conv=0), with_mixer(mask={"size": 0})):
        with pytest.raises(ValueError):
            config_from_dict(bad)
    c = json.loads(json.dumps(base))
    c["layers"][0]["type"] = "other"
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

    cfg = config_from_dict(U.CONFIGS["mixed"])
    w = {k: v.to(torch.bfloat16).contiguous() for k, v in U.weights("mixed").items()}
    layout = make_layout(cfg)
    for breakage in ("missing", "shape", "extra"):
        p = tmp_path / breakage
        p.mkdir()
        x = dict(w)
        if breakage == "missing":
            del x["l0.mix.talk"]
        elif breakage == "shape":
            x["l0.mix.q"] = x["l0.mix.q"][:-1].contiguous()
        else:
            x["l1.mlp.gate"] = torch.zeros(3, 3, dtype=torch.bfloat16)  # that layer has no feed-forward
        save_file(x, str(p / "model.safetensors"))
        with pytest.raises((KeyError, ValueError)):
            ckpt.load_hf_model(str(p), layout)


def test_random_init_clears_padding():
    cfg = PRESETS["dezelorn-tiny"]
    layout = make_layout(cfg)
    flat = torch.empty(layout.total)
    layout.init_random_(flat, 3)
    dev = torch.empty(layout.total)
    layout.init_random_device_(dev, 3)
    for f in (flat, dev):
        assert 0 < int((f != 0).sum()) <= cfg.num_parameters()
        assert float(layout.view(f, "layers.0.talk").diagonal().mean()) > 0.9


def test_step_tables():
    flat, where = host_batch([(3, 5, np.arange(130)), (1, 0, np.asarray([7, 8]))], [4, 1, 4], 1000)
    ids, sb = split_batch(torch.from_numpy(flat), where, torch.zeros(4, 4, dtype=torch.int32))
    assert sb.T == 132 and ids.tolist() == list(range(130)) + [7, 8]
    assert sb.rows[0].tolist() == [3, 5, 0, 0] and sb.rows[129].tolist() == [3, 134, 0, 0] and sb.rows[131].tolist() == [1, 1, 130, 0]
    assert {k: v.tolist() for k, v in sb.ring_rows.items()} == {1: [129, 131], 4: [126, 127, 128, 129, 130, 131]}
    assert sorted(map(tuple, sb.tiles.tolist())) == [(0, 128, 5, 0), (128, 2, 133, 0), (130, 2, 0, 144)]
    assert sb.pages.tolist() == [[3, p] for p in range(9)] + [[1, 0]]
    _, near = split_batch(*[f(x) for f, x in zip((torch.from_numpy, lambda w: w), host_batch([(2, 100, np.arange(3))], [1], 20))], None)
    assert near.pages.tolist() == [[2, 5], [2, 6]] and near.tiles.tolist() == [[0, 3, 100, -80]]
    assert sb.rows.storage_offset() % 4 == 0 and sb.tiles.storage_offset() % 4 == 0


def _sched(**kw):
    from async_grpo_nccl_b200.ops import native

    args = dict(num_blocks=32, block_size=16, max_seqs=4, max_blocks_per_seq=16, max_prefill_tokens=256)
    args.update(kw)
    return native().Scheduler(**args)


def test_scheduler_step_wise_sequences():
    s = _sched()
    a, slot_a = s.open_seq()
    b, slot_b = s.open_seq()
    assert slot_a != slot_b and s.num_running == 0 and s.num_free_slots == 2
    up = s.extend_seq(a, 17)
    assert [u[:2] for u in up] == [(slot_a, 0), (slot_a, 1)] and s.extend_seq(a, 15) == []
    assert len(s.extend_seq(a, 1)) == 1 and s.seq_info(a)["len"] == 33
    s.extend_seq(b, 5)
    plan = s.plan_decode()  # does not advance sequences that the caller drives
    assert plan["num_active"] == 0 and s.seq_info(a)["len"] == 33
    free = s.num_free_blocks
    s.finish(a)
    assert s.num_free_blocks == free + 3 and s.num_free_slots == 3
    with pytest.raises(RuntimeError):
        s.extend_seq(a, 1)
    with pytest.raises(RuntimeError):
        s.extend_seq(b, 16 * 16)
    s.finish(b)
    assert s.num_free_blocks == 32


def test_scheduler_gives_back_blocks_outside_the_window():
    s = _sched(window_tokens=20)
    a, _ = s.open_seq()
    total = 0
    for n in (1, 40, 2, 3, 60, 1, 1):
        s.extend_seq(a, n)
        total += n
        blocks = s.seq_info(a)["blocks"]
        first = max(0, total - n - 20 + 1) // 16   # oldest key that the first token of this step sees
        assert all(x == -1 for x in blocks[:first]) and all(x >= 0 for x in blocks[first:])
        assert s.num_free_blocks == 32 - (len(blocks) - first)
    s.finish(a)
    assert s.num_free_blocks == 32
    # the same while decoding; two samples share a prompt's blocks until each has moved on
    s.add_group(7, 33, 2, 100)
    p = s.plan_prefill()
    assert len(p["seq_ids"]) == 2
    for step in range(80):
        plan = s.plan_decode()
        assert plan["num_active"] == 2
    for q in p["seq_ids"]:
        blocks = s.seq_info(q)["blocks"]
        assert sum(x >= 0 for x in blocks) <= 3
        s.finish(q)
    assert s.num_free_blocks == 32


def test_generate_command_line_reads_prompts(tmp_path):
    import argparse

    from async_grpo_nccl_b200.generate import read_prompts

    f = tmp_path / "p.jsonl"
    f.write_text(json.dumps({"input_token_ids": [4, 5]}) + "\n\n" + json.dumps({"input_token_ids": [6]}) + "\n")
    got = read_prompts(argparse.Namespace(prompt_ids=["1,2,3"], prompt=[], prompts=str(f)), None)
    assert got == [[1, 2, 3], [4, 5], [6]]
    with pytest.raises(SystemExit):
        read_prompts(argparse.Namespace(prompt_ids=[], prompt=["hi"], prompts=None), None)


# ---- the oracle's own mechanisms on cases that can be worked out by hand ----
def test_oracle_mechanisms():
    u = torch.tensor([[1.0], [10.0], [100.0]], dtype=torch.float64)
    assert O.short_conv(u, torch.tensor([[2.0, 3.0]], dtype=torch.float64)).flatten().tolist() == [3.0, 32.0, 320.0]
    assert O.query_temperature(6, 1.0, 3, torch.float64)[:2].tolist() == [1.0, 1.0]
    assert float(O.query_temperature(6, 1.0, 3, torch.float64)[2]) == pytest.approx(1 + np.log(2))
    assert O.window_mask(4, 2).int().tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    w = torch.rand(2, 3, 3, dtype=torch.float64)
    mixed = O.mix_heads(w, torch.tensor([[0.0, 1.0], [1.0, 1.0]], dtype=torch.float64))
    assert torch.allclose(mixed[0], w[1]) and torch.allclose(mixed[1], w[0] + w[1])


def test_a_planted_mistake_shows_in_the_oracle():
    """Each mechanism left out (or off by one) changes the oracle's logits by far more than the tests' tolerances."""
    name, n = "odd", 60
    base, cfg, w, t = U.oracle_logits(name, n), U.CONFIGS[name], U.weights(name), U.tokens(name, n)

    def changed(mutate_cfg=None, mutate_w=None):
        c, x = json.loads(json.dumps(cfg)), dict(w)
        if mutate_cfg:
            for l in c["layers"]:
                mutate_cfg(l["mixer"])
        if mutate_w:
            for k in list(x):
                x[k] = mutate_w(k, x[k])
        return U.rel_rms(O.forward(c, x, t), base)

    assert changed(lambda m: m["q_temp"].update(coef=0.0)) > 0.05
    assert changed(lambda m: m["mask"].update(size=m["mask"]["size"] - 1)) > 1e-3   # only the last rows, one key each
    assert changed(mutate_w=lambda k, v: torch.eye(6, dtype=v.dtype) if k.endswith("talk") else v) > 0.05
    assert changed(mutate_w=lambda k, v: v * 0 if k.endswith("r1") else v) > 0.05
    assert changed(mutate_w=lambda k, v: v * torch.tensor([0.0, 1, 1]) if k.endswith("conv") else v) > 0.05
    assert changed(mutate_w=lambda k, v: v * 0 if k.endswith(".b") else v) > 0.05
