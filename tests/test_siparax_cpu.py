"""Siparax through the library's own cache, step function and generation loop on a CPU (the kernels' meaning restated
in torch, tests/emulated_ops.py), against the plain implementation: what is tested here is the host side, i.e. the
configuration, the cache entries (latent rows that several layers read, the delta rule's state and its convolution's
record), and the cutting of work into steps."""

import copy
import json

import pytest
import torch

import siparax_cases as cases
from conftest import random_tokens
from emulated_ops import EmulatedOps
from helpers import assert_close, run_ragged_batches, run_tail_by_one, run_whole
from plain import siparax_plain as plain
from starter_b200.cache import KVGroup, StateGroup
from starter_b200.config import ConfigError, config_from_dict, load_config
from starter_b200.engine import Engine
from starter_b200.engine.session import Session


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: cases.write_folder(name, tmp_path_factory.mktemp(f"siparax_{name}"), dtype=torch.float32) for name in cases.CASES}


def session(folder, **kw):
    args = dict(dtype="float32", device="cpu", ops=EmulatedOps(), max_tokens=64 * 12, max_seqs=4)
    args.update(kw)
    return Session(folder, **args)


def test_configuration_round_trip_and_parts(folders):
    cfg = load_config(folders["A"])
    assert cfg.architecture == "Siparax" and config_from_dict(cfg.to_dict()) == cfg
    spec = cfg.model_spec()
    assert spec.residual_float32 and not spec.tie_embeddings and spec.logit_softcap == 12.0
    assert (spec.embedding_norm.kind, spec.final_norm.kind, spec.final_norm.eps) == ("layernorm", "layernorm", 1e-5)
    assert [b.kind for b in spec.layers] == ["prenorm"] * 5 and [b.ff is None for b in spec.layers] == [False, False, True, False, False]
    assert {b.ff.activation for b in spec.layers if b.ff is not None} == {"gelu_tanh"}
    assert [b.mixer.kind for b in spec.layers] == ["latent_attention", "channel_delta", "latent_attention", "latent_attention", "latent_attention"]
    assert [b.mixer.position.kind for b in spec.layers if b.mixer.kind == "latent_attention"] == \
        ["rope_half_scaled", "rope_half_scaled", "rope_pairs", "rope_half_scaled"]
    assert [(b.mixer.head_gate, b.mixer.kv_from) for b in spec.layers if b.mixer.kind == "latent_attention"] == \
        [(True, None), (True, 0), (False, None), (True, 0)]
    m = spec.layers[3].mixer
    assert (m.num_heads, m.head_dim, m.rot_dim, m.v_dim, m.q_rank, m.kv_rank) == (5, 24, 12, 20, 28, 44)
    assert (m.position.theta, m.position.rotary_dim, m.position.factor, m.position.original, m.position.fast, m.position.slow) == \
        (500.0, 12, 2.0, 40.0, 6.0, 1.0)
    d = spec.layers[1].mixer
    assert (d.num_heads, d.num_kv_heads, d.head_dim, d.v_dim, d.taps, d.decay_rank, d.gate_rank) == (6, 2, 16, 24, 3, 20, 12)
    names = cfg.tensor_names()
    assert names.embedding_norm == {"weight": "embed.norm", "bias": "embed.norm.b"} and names.final_norm["bias"] == "final.norm.b"
    assert names.layers[0]["mixer"]["g"] == "l0.mix.g" and "g" not in names.layers[3]["mixer"] and "dkv" not in names.layers[2]["mixer"]
    assert names.layers[1]["mixer"]["k_conv"] == "l1.mix.k.conv" and names.layers[0]["ff_norm"]["bias"] == "l0.norm2.b"
    assert "ff" not in names.layers[2]
    bare = cases.config("C").model_spec()
    assert bare.logit_softcap is None and bare.layers[1].mixer.position.factor is None


def test_inner_sizes_come_from_the_tensors_shapes(folders):
    raw = copy.deepcopy(cases.CASES["A"])
    del raw["layers"][1]["mixer"]["decay_rank"], raw["layers"][1]["mixer"]["gate_rank"]
    cfg = config_from_dict(raw)
    with pytest.raises(ConfigError, match="shapes"):
        cfg.model_spec()
    m = cfg.with_shapes({"l1.mix.a1": (20, 96), "l1.mix.g1": (12, 96)}).model_spec().layers[1].mixer
    assert (m.decay_rank, m.gate_rank) == (20, 12)


@pytest.mark.parametrize("change, what", [
    (lambda r: r["layers"][0].update(type="attention"), "unknown"),
    (lambda r: r["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda r: r["layers"][1]["mixer"].update(kv_heads=4), "evenly"),
    (lambda r: r["layers"][1]["mixer"].update(conv=0), "conv"),
    (lambda r: r["layers"][0]["mixer"]["rot"].update(dims=7), "even"),
    (lambda r: r["layers"][0]["mixer"]["rot"].update(dims=10), "at most rot_dim"),
    (lambda r: r["layers"][0]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda r: r["layers"][2]["mixer"].update(kv_from=2), "earlier layer"),
    (lambda r: r["layers"][2]["mixer"].update(kv_from=1), "makes no latents"),
    (lambda r: r["layers"][4]["mixer"].update(kv_from=2), "makes no latents"),
    (lambda r: r["layers"][4]["mixer"].update(kv_rank=44), "makes no latents"),
    (lambda r: r["layers"][1]["mixer"].update(kv_from=0), "earlier layer"),
    (lambda r: r["layers"][0]["mlp"].update(kind="moe"), "not built"),
    (lambda r: r.update(logit_softcap=0.0), "positive"),
    (lambda r: r.pop("norm"), "norm"),
])
def test_bad_configurations_are_refused(change, what):
    raw = copy.deepcopy(cases.CASES["A"])
    change(raw)
    with pytest.raises(ConfigError, match=what):
        config_from_dict(raw)


def test_cache_entries(folders):
    layers = session(folders["A"]).cache.layers
    assert isinstance(layers[0].group, KVGroup) and layers[0].group.k.shape[2:] == (1, 64, 48 + 8) and layers[0].group.v is None
    assert layers[2] is layers[0] and layers[4] is layers[0] and layers[3] is not layers[0]     # readers hold no rows of their own
    assert layers[3].group.k.shape[2:] == (1, 64, 44 + 12)
    assert isinstance(layers[1].group, StateGroup) and layers[1].state.shape[1:] == (6 * 16 * 24,)
    assert layers[1].aux.state.shape[1:] == (2, 2 * 2 * 16 + 6 * 24) and layers[1].aux.aux is None
    assert all(l.state.dtype == torch.float32 for l in (layers[1], layers[1].aux))
    bare = session(folders["C"]).cache.layers
    assert bare[0].aux is None and bare[3].aux.state.shape[1:] == (4, 2 * 136 + 2 * 130)        # one tap keeps no record


@pytest.mark.parametrize("name", list(cases.CASES))
def test_every_cutting_matches_plain(folders, name):
    folder = folders[name]
    seqs = random_tokens(cases.CASES[name]["vocab"], (5, 90, 41, 1, 64, 65, 2), seed=3)
    ref = cases.plain_logits(folder, seqs)
    sess = session(folder, max_rows=50)     # a step of more than 50 rows goes through in several forward passes
    assert_close(run_whole(sess, seqs), ref, "float32", "alone and whole")
    assert_close(run_whole(sess, seqs[:3], together=True), ref[:3], "float32", "one ragged step")
    assert_close(run_tail_by_one(sess, seqs, tail=30), ref, "float32", "tail one by one")
    assert_close(run_ragged_batches(sess, seqs, batch_size=3, poison=True), ref, "float32", "ragged batches, freed pages poisoned")
    assert sess.cache.slots.n_held == 0


def test_a_whole_prompt_in_the_narrow_form(folders):
    """One sequence's first step of 64 rows and more: the readers take the rows that wait in the step's scratch."""
    seqs = random_tokens(211, (64, 150, 63), seed=14)
    assert_close(run_whole(session(folders["A"]), seqs), cases.plain_logits(folders["A"], seqs), "float32", "one step each")


def test_portions_down_to_two_tokens(folders):
    seqs = random_tokens(211, (37,), seed=4)
    ref = cases.plain_logits(folders["A"], seqs)
    for portion in (2, 3, 7, 20, 21):
        sess = session(folders["A"], max_rows=portion)
        assert_close(run_whole(sess, seqs), ref, "float32", f"portions of {portion}")


def test_state_of_a_freed_slot_does_not_leak(folders):
    """A slot that held a sequence is used again: convolutions and state start from zeros."""
    sess = session(folders["D"], max_seqs=1)
    seqs = random_tokens(64, (70, 9, 3), seed=5)
    ref = cases.plain_logits(folders["D"], seqs)
    assert_close(run_whole(sess, seqs), ref, "float32", "later sequences in the first one's slot")
    assert_close(run_tail_by_one(sess, seqs, tail=8), ref, "float32", "and decoded")


def test_layers_match_plain(folders):
    """The residual after every layer, taken from the library's own stream."""
    cfg, tensors = plain.read_folder(folders["A"])
    tokens = random_tokens(211, (19,), seed=9)[0]
    want = []
    plain.forward(cfg, tensors, tokens, want)
    sess = session(folders["A"])
    seen = []
    for block in sess.model.blocks:
        inner = block.forward

        def spy(ctx, stream, layer_cache, inner=inner):
            inner(ctx, stream, layer_cache)
            seen.append(stream.x + (stream.pending if stream.pending is not None else 0.0))
        block.forward = spy
    run_whole(sess, [tokens])
    assert len(seen) == len(want) == 5
    for i, (got, ref) in enumerate(zip(seen, want)):
        assert got.dtype == torch.float32
        assert float((got - ref).abs().max()) <= 1e-4 * float(ref.abs().max()), f"layer {i}"


def test_greedy_generation_through_the_entry_point(folders):
    cfg, tensors = plain.read_folder(folders["C"])
    prompts = random_tokens(97, (3, 11, 1), seed=6)
    want = plain.generate(cfg, tensors, prompts, 10)
    engine = Engine.from_session(session(folders["C"]), use_graphs=False)
    assert engine.generate_all(prompts, 10) == want
    assert engine.session.cache.slots.n_held == 0


def test_random_weights_from_the_command_line(tmp_path):
    from starter_b200.cli import main
    (tmp_path / "config.json").write_text(json.dumps(cases.CASES["D"]))
    assert main(["random-weights", "--config", str(tmp_path / "config.json"), "--seed", "3", "--out", str(tmp_path / "model")]) == 0
    sess = session(tmp_path / "model")
    assert sess.model.spec.vocab_size == 64 and len(sess.model.blocks) == 5
    seqs = random_tokens(64, (12,), seed=8)
    assert_close(run_whole(sess, seqs), cases.plain_logits(tmp_path / "model", seqs), "float32", "folder from the command line")
