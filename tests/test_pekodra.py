"""The Pekodra decoder in the engine against the plain float64 statement of it (``plain_pekodra``).

Small configurations of the tests' own, random weights shaped so that faults show (peaked attention, norm weights and
biases that are not small, routers whose logits spread), and every way of cutting and batching. The same tests run on a
CPU with the plain PyTorch statements of the kernels (host logic: pages behind a window, the caches of a layer that runs
several times) and, marked ``gpu``, with the compiled kernels in float32 and bfloat16. The kernels' new options are also
compared one by one with their plain statements.
"""

import json
import math
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import plain_pekodra as plain
import traces

from tiny_pekodra import (ATT, ATT_BARE, ATT_EVEN, ATT_EVEN32, ATT_EVEN64, ATT_FULL, ATT_ODD, ATT_SELF, BLEND, CONFIGS, LENGTHS, PAGE, TOL, attn, dense, layer,
                          make_folder, model, moe, plant, prompts)

ROOT = Path(__file__).resolve().parent.parent
# A routing margin (the gap between two logits, which are a few units large) below this may fall the other way: in
# bfloat16 through the rounding of the router's input and of the layers before it, in float32 through the order of sums.
CLOSE_CALL = {"float32": 1e-3, "bfloat16": 0.2}


def runner_for(folder, dtype, device, page, max_tokens, ops=None, max_requests=4, context=None, **kw):
    from akas_b200.config import EngineConfig
    from akas_b200.engine.runner import ModelRunner

    cfg = EngineConfig(dtype=dtype, device=device, page_size=page, max_tokens=max_tokens, max_requests=max_requests,
                       context=context or max_tokens, cuda_graphs=False, **kw)
    return ModelRunner(folder, cfg, ops=ops)


def oracle(config, w, tokens):
    """(logits [T, vocab], margin [T]): the least routing margin of a position over all routed layer runs; where it is
    a close call, the engine may decide the other way (and every later position may feel it through the mixers)."""
    margins = []
    logits = plain.forward(tokens, w, config, margins=margins).numpy()
    least = np.full(len(tokens), np.inf)
    for per_layer in margins:
        least = np.minimum(least, np.asarray(per_layer))
    return logits, least


def compare(got, want, dtype, what):
    for rid, (logits, least) in want.items():
        rows = np.nonzero(least >= CLOSE_CALL[dtype])[0]
        if dtype != "float32":
            error = np.abs(got[rid] - logits).max(axis=-1) / np.abs(logits).max()
            assert np.median(error) <= 0.5 * TOL[dtype], f"{what}: request {rid}: median error {np.median(error):.3g}"
            if len(rows) == 0:
                continue
        bad = traces.first_bad(got[rid][rows], logits[rows], TOL[dtype])
        assert bad is None, (f"{what}: request {rid} first differs at position {rows[bad]} "
                             f"{traces.worst(got[rid][rows], logits[rows])}")


def run_modes(key, dtype, device, ops, tmp_path, modes):
    config = CONFIGS[key]
    folder, w = make_folder(config, seed=31, folder=tmp_path / key)
    reqs = {f"r{i}": p for i, p in enumerate(prompts(config["vocab"], LENGTHS[key], seed=6))}
    want = {rid: oracle(config, w, toks) for rid, toks in reqs.items()}
    page = PAGE[key]
    longest = -(-max(len(t) for t in reqs.values()) // page) * page
    for mode in modes:
        if mode == "mixed":
            steps, peak = traces.mixed(reqs, {rid: max(1, len(t) - 9) for rid, t in reqs.items()}, seed=3, live=3, page=page)
            runner = runner_for(folder, dtype, device, page, peak, ops, max_requests=3, context=longest)
        else:
            steps = getattr(traces, mode)(reqs)
            runner = runner_for(folder, dtype, device, page, longest, ops, max_requests=2)
        got = traces.replay(runner, steps)
        assert not runner.cache.live() and runner.cache.min_free_pages() == runner.cache.num_pages
        compare(got, want, dtype, f"{key}/{dtype}/{mode}")


MODES = ["whole", "tail_decoded", "portions", "mixed"]


@pytest.mark.parametrize("key", list(CONFIGS))
def test_every_way_of_cutting_on_the_plain_operations(key, tmp_path):
    from akas_b200.ops import reference

    run_modes(key, "float32", "cpu", reference, tmp_path, MODES)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", list(CONFIGS))
def test_every_way_of_cutting_on_the_kernels(key, dtype, tmp_path):
    run_modes(key, dtype, "cuda:0", None, tmp_path, MODES)


def test_config_round_trip_registry_and_inventory(tmp_path):
    from akas_b200.config import ConfigError, PekodraConfig, config_from_dict, load_config
    from akas_b200.engine.runner import kernel_kinds
    from akas_b200.ops import reference
    from akas_b200.weights.loader import WeightError

    config = config_from_dict(CONFIGS["mix"])
    assert isinstance(config, PekodraConfig) and config_from_dict(config.to_dict()) == config
    assert config_from_dict(json.loads(json.dumps(config.to_dict()))) == config
    spec = config.model_spec()
    # layers 1..3 three times in a row, each run with a cache of its own; the embedding joins in front of every pass
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4]
    assert [i for i, e in enumerate(spec.schedule) if e.join == "loop.in"] == [1, 4, 7] and all(e.cache is None for e in spec.schedule)
    assert not any(e.add_embedding for e in spec.schedule)
    assert all(l.arrangement == "parallel" and l.mixer_norm.zero_centered and l.mixer_norm.eps == 1e-5 for l in spec.layers)
    first, second, fourth = spec.layers[0], spec.layers[1], spec.layers[3]
    assert first.mixer.qk_unit_eps == 1e-5 and first.mixer.window == 21 and first.mixer.value_dim == 16 and first.mixer.general
    assert first.mixer.position.blend == (6.0, 48.0, 8.0, 0.5) and first.mixer.position.amplitude == pytest.approx(0.1 * math.log(6.0) + 1.0)
    assert first.mixer.position.rotary == 16 and first.mixer.scale == 0.5 and fourth.mixer.position is None and fourth.ffn is None
    assert (first.ffn.scoring, first.ffn.renormalize, first.ffn.correction, first.ffn.gated) == ("softmax", True, False, False)
    assert first.ffn.activation == "relu2" and first.ffn.top == 2 and first.ffn.shared_size == 40 and not first.ffn.shared_gate
    assert second.ffn.kind == "gated_mlp" and second.ffn.activation == "gelu_tanh" and second.ffn.bias and second.ffn.intermediate_size == 48
    assert spec.head_name == "head" and spec.logit_scale == 0.7 and spec.embedding_multiplier == 3.0
    assert set(kernel_kinds(spec)) == {"attention_general", "rope", "moe"}
    # values of the keys' size, at sizes that the kernels for plain attention take: those, whatever the norm's place
    even = config_from_dict(CONFIGS["even"]).model_spec()
    assert not any(l.mixer.general for l in even.layers) and set(kernel_kinds(even)) == {"attention", "moe"}
    assert config_from_dict(CONFIGS["alone"]).loop is None
    folder, _ = make_folder(CONFIGS["odd"], seed=1, folder=tmp_path / "m")
    assert load_config(folder) == config_from_dict(CONFIGS["odd"])
    for change, message in ((lambda c: c["layers"][0]["mixer"].update(kv_heads=2), "kv_heads"),
                            (lambda c: c["layers"][0]["mixer"].update(mask=dict(size=0)), "size"),
                            (lambda c: c["layers"][0]["mixer"].pop("mask"), "mask"),
                            (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=5), "rot.dims"),
                            (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=22), "rot.dims"),
                            (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
                            (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "top"),
                            (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "kind"),
                            (lambda c: c["loop"].update(stop=7), "loop"),
                            (lambda c: c["loop"].update(times=0), "times"),
                            (lambda c: c["layers"][0].update(type="retention"), "type")):
        broken = json.loads(json.dumps(CONFIGS["odd"]))
        change(broken)
        with pytest.raises(ConfigError, match=message):
            config_from_dict(broken)
    # a checkpoint without the joining matrix, or with a tensor the design does not have, is refused
    from safetensors.torch import load_file, save_file

    tensors = load_file(str(folder / "model.safetensors"))
    assert tensors["loop.in"].shape == (52, 104) and tensors["l0.mlp.shared.up"].shape == (12, 52) and "l0.mlp.e0.gate" not in tensors
    assert tensors["l1.mlp.down.b"].shape == (52,) and "l2.norm2" not in tensors and "l3.mlp.shared.up" not in tensors
    del tensors["loop.in"]
    tensors["l1.mix.q.b"] = torch.ones(96, dtype=torch.bfloat16)
    tensors["l2.norm2"] = torch.zeros(52, dtype=torch.bfloat16)  # the norm that a feed-forward would have: may lie about
    save_file(tensors, str(folder / "model.safetensors"))
    with pytest.raises(WeightError, match="loop.in") as caught:
        runner_for(folder, "float32", "cpu", 8, 64, reference)
    assert "l1.mix.q.b" in str(caught.value) and "l2.norm2" not in str(caught.value)


# --------------------------------------------------------------------------- each mechanism alone


def one_mechanism(config, tmp_path, seed=5, length=60):
    """The engine on the plain operations against the oracle for a small model that isolates a mechanism."""
    from akas_b200.ops import reference

    folder, w = make_folder(config, seed=seed, folder=tmp_path / "one")
    toks = prompts(config["vocab"], [length], seed=seed)[0]
    runner = runner_for(folder, "float32", "cpu", 8, -(-length // 8) * 8, reference)
    got = traces.replay(runner, traces.portions({"a": toks}, sizes=(9, 1, 2, 17)))["a"]
    want = plain.forward(toks, w, config).numpy()
    assert traces.first_bad(got, want, TOL["float32"]) is None, traces.worst(got, want)
    return w, toks, want


def test_two_norms_of_the_same_rows():
    from akas_b200.ops import reference

    g = torch.Generator().manual_seed(3)
    x, w1, w2 = torch.randn(7, 20, generator=g) * 4, torch.randn(20, generator=g), torch.randn(20, generator=g)
    a, b = reference.rmsnorm_pair(x, w1, w2, 1e-3, True, torch.float32)
    assert (a.double() - plain.norm(x.double(), w1.double(), 1e-3)).abs().max() < 1e-5
    assert (b.double() - plain.norm(x.double(), w2.double(), 1e-3)).abs().max() < 1e-5
    assert (plain.norm(torch.zeros(1, 4, dtype=plain.F), torch.ones(4, dtype=plain.F), 1e-3) == 0).all()


def test_rotary_rates_blended():
    """The rates the engine's rotation is built with against the oracle's: plain, blended with the edges inside the
    pairs, outside them, and both at the first pair."""
    from akas_b200.config import config_from_dict
    from akas_b200.parts.base import Runtime
    from akas_b200.parts.rope import Rope

    rt = Runtime(torch.float32, torch.device("cpu"), None)
    for rot in (dict(base=10000.0, dims=16), dict(base=300.0, dims=16, scaling=BLEND),
                dict(base=400000.0, dims=32, scaling=dict(factor=4.0, original=1024, fast=16.0, slow=2.0)),
                dict(base=50.0, dims=6, scaling=dict(factor=3.0, original=4000, fast=2.0, slow=1.0)),
                dict(base=1e6, dims=8, scaling=dict(factor=5.0, original=2, fast=64.0, slow=32.0)),
                dict(base=10000.0, dims=64, scaling=dict(factor=1.0, original=100, fast=32.0, slow=1.0))):
        spec = config_from_dict(model(8, 8, [layer(dict(ATT, dim=64, rot=rot), None)])).model_spec().layers[0].mixer.position
        rope = Rope(spec, rt)
        want, amp = plain.rates(rot)
        assert np.allclose(rope.inv_freq.numpy(), np.asarray(want), rtol=1e-12, atol=0.0), rot
        assert rope.amplitude == pytest.approx(amp, rel=1e-12)
    slowed, bare = plain.rates(dict(base=300.0, dims=16, scaling=BLEND))[0], plain.rates(dict(base=300.0, dims=16))[0]
    assert slowed[0] == bare[0] and slowed[7] == pytest.approx(bare[7] / 6.0) and bare[2] / 6.0 < slowed[2] < bare[2]


def _unit_case(heads, kv_heads, dim, vdim, rot, page, n=37, seed=0):
    g = torch.Generator().manual_seed(seed + dim)
    q, k, v = (torch.randn(n, width, generator=g) * 2 for width in (heads * dim, kv_heads * dim, kv_heads * vdim))
    pages = -(-n // page)
    table = torch.randperm(pages, generator=g).to(torch.int32)[None]
    return q, k, v, table, torch.zeros(n, dtype=torch.int32), torch.arange(n, dtype=torch.int32), pages


def test_unit_heads_behind_the_rotation():
    """q and k through the operation against the oracle: rotation first, then every head over its root mean square; a
    rotation of a part of the head with an amplitude changes what the division sees, so the other order differs."""
    from akas_b200.ops import reference

    rot = dict(base=300.0, dims=16, scaling=BLEND)
    q, k, v, table, seq, pos, pages = _unit_case(4, 2, 24, 16, rot, 8)
    want = plain.rms(plain.rotate(q.double().reshape(37, 4, 24), rot), 1e-4)
    freq, amp = plain.rates(rot)
    cos, sin = reference.rope_tables(pos, torch.tensor(freq, dtype=torch.float64), amp)
    k_pool, v_pool = torch.zeros(pages, 2, 8, 24), torch.zeros(pages, 2, 8, 16)
    got = reference.qk_norm_store(q, k, v, 4, 2, 24, 16, None, None, 0.0, k_pool, v_pool, table, seq, pos, 8, cos=cos, sin=sin, unit_eps=1e-4)
    assert (got.double().reshape(37, 4, 24) - want).abs().max() < 1e-5
    stored = k_pool[table[0].long()].permute(0, 2, 1, 3).reshape(-1, 2, 24)[:37]
    assert (stored.double() - plain.rms(plain.rotate(k.double().reshape(37, 2, 24), rot), 1e-4)).abs().max() < 1e-5
    other = plain.rotate(plain.rms(q.double().reshape(37, 4, 24), 1e-4), rot)
    assert (other - want).abs().max() > 1e-2
    assert torch.allclose((want * want).mean(-1), torch.ones(37, 4, dtype=plain.F), atol=1e-3)


@pytest.mark.parametrize("mixer", [ATT, ATT_FULL, ATT_ODD, ATT_SELF, ATT_BARE, ATT_EVEN, ATT_EVEN32, ATT_EVEN64])
def test_attention_alone(mixer, tmp_path):
    one_mechanism(model(48, 60, [layer(mixer, None)]), tmp_path)


def test_feed_forwards_alone(tmp_path):
    """Dense; routed with one and with several experts a token, with and without the expert that every token passes; as
    many experts a token as there are; and the router's rule on the oracle."""
    for i, mlp in enumerate((dense(40), moe(16, 5, 1), moe(24, 6, 2, shared=40), moe(8, 3, 3, shared=8), moe(12, 1, 1))):
        w, _, _ = one_mechanism(model(48, 60, [layer(ATT_SELF, mlp)]), tmp_path / str(i))
        if i == 2:
            kept = w
    h = torch.randn(9, 48, dtype=torch.float64)
    wf = {k[len("l0.mlp."):]: v for k, v in kept.items() if k.startswith("l0.mlp.")}
    chosen, weights = plain.route(h, wf, "", dict(experts=6, top=2))
    assert np.allclose(weights.sum(-1).numpy(), 1.0)
    z = h @ wf["router"].T
    everything = torch.softmax(z, dim=-1)
    picked = torch.gather(everything, 1, chosen)
    assert np.allclose((picked / picked.sum(-1, keepdim=True)).numpy(), weights.numpy())  # over the chosen alone
    assert np.abs(picked.numpy() - weights.numpy()).max() > 1e-2


def test_both_sublayers_read_the_same_stream(tmp_path):
    """The feed-forward does not see what the mixer added: the oracle with the sublayers one after the other differs."""
    config = model(48, 60, [layer(ATT, dense(40))])
    w, toks, want = one_mechanism(config, tmp_path)
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(toks)] * config["embedding"]["scale"]
    x = x + plain.attention(plain.norm(x, w["l0.norm1"], eps), w, "l0.mix.", ATT, eps)
    x = x + plain.dense(plain.norm(x, w["l0.norm2"], eps), w, "l0.mlp.")
    serial = (plain.norm(x, w["final.norm"], eps) @ w["head"].T * config["logit_scale"]).numpy()
    assert np.abs(serial - want).max() > 1e-2 * np.abs(want).max()


def test_a_block_with_scales_and_a_norm_for_each_sublayer():
    """The arrangement's other options beside two norms: a learned scale per sublayer and a constant, and a feed-forward
    that has no halves; against the same sums written out."""
    from akas_b200.config import GatedMLPSpec, LayerSpec, MLPSpec, RMSNormSpec
    from akas_b200.ops import reference
    from akas_b200.parts.base import Mixer, Runtime, register_mixer
    from akas_b200.parts.block import Block

    class Double(Mixer):
        def forward(self, x, ctx, cache=None, residual=None, write=True):
            out = 2.0 * x.to(torch.float32)
            return out if residual is None else residual.add_(out)

    register_mixer("test_double", Double)

    class Spec:
        kind = "test_double"

    rt = Runtime(torch.float32, torch.device("cpu"), reference)
    g = torch.Generator().manual_seed(2)
    norm = RMSNormSpec(12, 1e-5, zero_centered=True)
    for ffn in (GatedMLPSpec(12, 20, bias=True), MLPSpec(12, 20)):
        for scaled in (False, True):
            spec = LayerSpec(Spec(), ffn, norm, norm, "m.", "f.", "n1", "n2", arrangement="parallel",
                             **(dict(residual_multiplier=0.5, mixer_scale_name="s1", ffn_scale_name="s2") if scaled else {}))
            block = Block(spec, rt)
            w = {k: torch.randn(p.shape, generator=g) * 0.5 for k, p in block.params().items()}
            block.load(lambda name: w[name])
            x = torch.randn(5, 12, generator=g)
            d = {k: v.double() for k, v in w.items()}
            n1, n2 = plain.norm(x.double(), d["n1"], 1e-5), plain.norm(x.double(), d["n2"], 1e-5)
            ff = plain.dense(n2, d, "f.") if ffn.kind == "gated_mlp" else torch.relu(n2 @ d["f.up"].T) ** 2 @ d["f.down"].T
            s1, s2, m = (d["s1"], d["s2"], 0.5) if scaled else (1.0, 1.0, 1.0)
            want = x.double() + m * (s1 * 2.0 * n1 + s2 * ff)
            got = block.forward(x.clone(), None)
            assert (got.double() - want).abs().max() < 1e-4 * want.abs().max(), (ffn.kind, scaled)


def test_the_loop_and_the_embedding_that_joins(tmp_path):
    """A loop of one pass joins the embedding once; every pass has a cache of its own and the embedding joins in front
    of each; what the embedding's half of the matrix holds is felt."""
    layers = [layer(ATT_SELF, dense(24)), layer(ATT, None), layer(ATT_ODD, moe(16, 4, 1, shared=8))]
    none = one_mechanism(model(48, 60, layers), tmp_path / "none")[2]
    w, toks, once = one_mechanism(model(48, 60, layers, loop=(0, 3, 1)), tmp_path / "once")
    thrice = model(48, 60, layers, loop=(1, 3, 3))
    _, _, many = one_mechanism(thrice, tmp_path / "thrice")
    assert plain.run_order(thrice) == [(0, False), (1, True), (2, False), (1, True), (2, False), (1, True), (2, False)]
    trace = []
    plain.forward(toks, w, thrice, trace)
    assert len(trace) == 7 and np.abs(many - once).max() > 1e-3 and np.abs(once - none).max() > 1e-3
    alone = dict(w)
    alone["loop.in"] = torch.cat([w["loop.in"][:, :48], torch.zeros(48, 48, dtype=torch.float64)], dim=1)
    assert np.abs(plain.forward(toks, alone, thrice).numpy() - many).max() > 1e-2 * np.abs(many).max()


# --------------------------------------------------------------------------- what a position sees


WINDOW = 130
KINDS = {"general": (dict(ATT, mask=dict(size=WINDOW), scale=1.0), 8),
         "plain": (dict(ATT_EVEN64, mask=dict(size=WINDOW), scale=0.3), 64), "plain, small pages": (dict(ATT_EVEN, mask=dict(size=WINDOW), scale=1.5), 8)}


def seen_case(device, dtype, ops, tmp_path, decode, kind):
    """One layer: the logits at position i change with the token at position j iff i - WINDOW < j <= i: just inside and
    just outside the window, keys at page borders, next to the query, the query itself; later tokens never; with the
    query in a prompt's portion or decoded alone."""
    from akas_b200.engine.batch import StepEntry

    i = 290
    mixer, page = KINDS[kind]
    config = model(48, 120, [layer(mixer, None)])
    folder, _ = make_folder(config, seed=44, folder=tmp_path / "edge")
    w = plant(folder, config, key_token=119, query_token=118)  # token 119 at position j is felt by token 118 at position i
    edge = i - WINDOW + 1
    cases = [(0, False), (1, False), (64, False), (edge - 2, False), (edge - 1, False), (edge, True), (edge + 1, True), (167, True),
             (168, True), (192, True), (255, True), (256, True), (i - 1, True), (i, True), (i + 1, False), (299, False)]
    base = prompts(118, [300], seed=9)[0]
    base[i] = 118

    def logits_at_i(tokens):
        runner = runner_for(folder, dtype, device, page, 320, ops)
        if decode:
            runner.step([StepEntry("a", tokens[:i], ())])
            out = runner.step([StepEntry("a", tokens[i:i + 1], (0,))])
        else:
            runner.step([StepEntry("a", tokens[:277], ())])
            out = runner.step([StepEntry("a", tokens[277:], (i - 277,))])
        return out.float().cpu().numpy()[0]

    ref = logits_at_i(base)
    for j, seen in cases:
        changed = list(base)
        changed[j] = 119 if j != i else 7
        got = logits_at_i(changed)
        diff = np.abs(got - ref).max()
        if seen:
            assert diff > 2e-2 * np.abs(ref).max(), f"position {i} does not see {j}"
        else:
            assert diff == 0.0, f"position {i} sees {j} (difference {diff})"
        if dtype == "float32" and seen:
            want = plain.forward(changed[: i + 1], w, config)[i].numpy()
            assert np.abs(got - want).max() <= TOL[dtype] * np.abs(want).max()


@pytest.mark.parametrize("kind", list(KINDS))
@pytest.mark.parametrize("decode", [False, True])
def test_what_a_position_sees_on_the_plain_operations(decode, kind, tmp_path):
    from akas_b200.ops import reference

    seen_case("cpu", "float32", reference, tmp_path, decode, kind)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", list(KINDS))
@pytest.mark.parametrize("decode", [False, True])
def test_what_a_position_sees_on_the_kernels(decode, dtype, kind, tmp_path):
    seen_case("cuda:0", dtype, None, tmp_path, decode, kind)


def far_key_case(device, dtype, ops, tmp_path, kind):
    """One key far back among hundreds is made to stand out, as the oldest one that the window still holds: the last
    position's attention must find it through scattered pages, in a portion and decoded alone, in every pass of a looped
    layer (each has its own pages); one position further back it must be gone."""
    from akas_b200.engine.batch import StepEntry

    mixer, page = KINDS[kind]
    config = model(48, 120, [layer(dict(mixer, mask=dict(size=497)), None)], loop=(0, 1, 2))
    folder, _ = make_folder(config, seed=47, folder=tmp_path / "far")
    w = plant(folder, config, key_token=119, query_token=118)
    toks = prompts(118, [500], seed=2)[0]
    toks[3], toks[-1] = 119, 118  # position 499 sees positions 3..499
    want = plain.forward(toks, w, config)[-1].numpy()
    moved = list(toks)
    moved[3], moved[2] = toks[2], 119
    past = plain.forward(moved, w, config)[-1].numpy()
    without = list(toks)
    without[3] = 5
    felt = np.abs(plain.forward(without, w, config)[-1].numpy() - want).max()
    assert felt > 0.1 * np.abs(want).max() and np.abs(past - want).max() > 0.1 * np.abs(want).max(), "the far key does not stand out"
    for tokens, expected in ((toks, want), (moved, past)):
        for cuts in ([500], [499, 1], [130, 70, 2, 290, 8]):
            runner = runner_for(folder, dtype, device, 2 * page, 640, ops, context=512) if page < 64 else \
                runner_for(folder, dtype, device, page, 640, ops, context=512)
            runner.admit("other")  # the request's pages are not the pool's first
            runner.cache.reserve("other", 40)
            at = 0
            for c in cuts:
                out = runner.step([StepEntry("a", tokens[at:at + c], (c - 1,) if at + c == 500 else ())])
                at += c
            got = out.float().cpu().numpy()[0]
            assert np.abs(got - expected).max() <= TOL[dtype] * np.abs(expected).max(), cuts


@pytest.mark.parametrize("kind", list(KINDS))
def test_a_far_key_is_found_on_the_plain_operations(kind, tmp_path):
    from akas_b200.ops import reference

    far_key_case("cpu", "float32", reference, tmp_path, kind)


@pytest.mark.gpu
@pytest.mark.parametrize("kind", list(KINDS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_key_is_found_on_the_kernels(dtype, kind, tmp_path):
    far_key_case("cuda:0", dtype, None, tmp_path, kind)


def test_freed_pages_are_used_again_and_not_read(tmp_path):
    """Two requests one after the other in a pool of one slot and just enough pages: the second gets the first one's
    pages (in every pass of the loop) and must compute as if it were alone."""
    from akas_b200.engine.batch import StepEntry
    from akas_b200.ops import reference

    config = CONFIGS["odd"]
    folder, w = make_folder(config, seed=12, folder=tmp_path / "m")
    a, b = prompts(config["vocab"], [30, 26], seed=5)
    runner = runner_for(folder, "float32", "cpu", 8, 32, reference, max_requests=1)
    runner.step([StepEntry("a", a, ())])
    runner.release("a")
    runner.step([StepEntry("b", b[:11], ())])
    got = runner.step([StepEntry("b", b[11:], tuple(range(15)))]).numpy()
    want = plain.forward(b, w, config).numpy()[11:]
    assert traces.first_bad(got, want, TOL["float32"]) is None, traces.worst(got, want)


def test_pages_behind_every_window_come_back_while_the_request_runs(tmp_path):
    """Layers with windows of different sizes keep different numbers of pages of a long request, and a page that one
    request left behind serves another one."""
    from akas_b200.engine.batch import StepEntry
    from akas_b200.ops import reference

    config = model(48, 60, [layer(dict(ATT, mask=dict(size=9)), None), layer(dict(ATT, mask=dict(size=40)), dense(16))], loop=(0, 2, 2))
    folder, w = make_folder(config, seed=12, folder=tmp_path / "m")
    a, b = prompts(60, [120, 50], seed=5)
    runner = runner_for(folder, "float32", "cpu", 8, 176, reference, max_requests=2, context=120)
    want = {"a": plain.forward(a, w, config).numpy(), "b": plain.forward(b, w, config).numpy()}
    at = {"a": 0, "b": 0}
    for step in range(60):
        entries = [StepEntry("a", a[at["a"]:at["a"] + 2], (0, 1))]
        if step >= 10 and at["b"] < len(b):
            entries.append(StepEntry("b", b[at["b"]:at["b"] + 1], (0,)))
        got = runner.step(entries).numpy()
        row = 0
        for e in entries:
            for k in range(len(e.tokens)):
                err = np.abs(got[row] - want[e.request][at[e.request] + k]).max() / np.abs(want[e.request]).max()
                assert err <= TOL["float32"], (step, e.request, k, err)
                row += 1
            at[e.request] += len(e.tokens)
        runner.cache.check()


def test_a_batch_of_unequal_requests_equals_each_alone(tmp_path):
    """A request's logits beside three others of other lengths, and alone."""
    from akas_b200.engine.batch import StepEntry
    from akas_b200.ops import reference

    config = CONFIGS["mix"]
    folder, _ = make_folder(config, seed=14, folder=tmp_path / "m")
    ps = prompts(config["vocab"], [1, 37, 2, 80], seed=5)
    runner = runner_for(folder, "float32", "cpu", 8, 256, reference)
    together = runner.step([StepEntry(i, p, (len(p) - 1,)) for i, p in enumerate(ps)]).numpy()
    for i, p in enumerate(ps):
        alone = runner_for(folder, "float32", "cpu", 8, 256, reference).step([StepEntry("x", p, (len(p) - 1,))]).numpy()
        assert np.abs(alone[0] - together[i]).max() <= 1e-5 * np.abs(alone).max()


# --------------------------------------------------------------------------- generation


def _greedy(config, w, prompt, count):
    toks = list(prompt)
    for _ in range(count):
        toks.append(int(plain.forward(toks, w, config)[-1].argmax()))
    return toks[len(prompt):]


def generation_case(device, dtype, ops, tmp_path, graphs):
    from akas_b200 import Engine, EngineConfig

    config = CONFIGS["mix"]
    folder, w = make_folder(config, seed=61, folder=tmp_path / "gen")
    ps = prompts(config["vocab"], [1, 9, 40, 23, 3], seed=8)
    cfg = EngineConfig(dtype=dtype, device=device, page_size=8, max_requests=3, context=128, max_tokens=1024, prefill_chunk=13,
                       prefill_requests=2, cuda_graphs=graphs)
    with Engine(str(folder), config=cfg, ops=ops) as engine:
        results = engine.generate(ps, max_tokens=10)
    for prompt, result in zip(ps, results):
        assert result["generated_tokens"] == _greedy(config, w, prompt, 10)


def test_greedy_generation_through_the_scheduler_on_the_plain_operations(tmp_path):
    from akas_b200.ops import reference

    generation_case("cpu", "float32", reference, tmp_path, False)


@pytest.mark.gpu
@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_scheduler_on_the_kernels(graphs, tmp_path):
    generation_case("cuda:0", "float32", None, tmp_path, graphs)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dtype, tmp_path):
    """200 decoded tokens for three requests of different lengths through captured graphs, against one whole pass of
    the plain model."""
    from akas_b200 import Engine, EngineConfig, StepEntry

    config = CONFIGS["mix"]
    folder, w = make_folder(config, seed=71, folder=tmp_path / "long")
    ps = prompts(config["vocab"], [5, 70, 33], seed=3)
    feed = prompts(config["vocab"], [200, 200, 200], seed=4)
    cfg = EngineConfig(dtype=dtype, device="cuda:0", page_size=8, max_requests=4, context=512, max_tokens=2048)
    with Engine(str(folder), config=cfg) as engine:
        runner = engine.runner
        runner.step([StepEntry(i, p, ()) for i, p in enumerate(ps)])
        rows = [[] for _ in ps]
        for t in range(200):
            logits = runner.step([StepEntry(i, (feed[i][t],), (0,)) for i in range(3)]).float().cpu().numpy()
            for i in range(3):
                rows[i].append(logits[i])
        assert 4 in runner._graphs
    want = {}
    for i, p in enumerate(ps):
        logits, least = oracle(config, w, p + feed[i])
        want[i] = (logits[len(p):], least[len(p):])
    compare({i: np.stack(r) for i, r in enumerate(rows)}, want, dtype, f"long decoding/{dtype}")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_program(dtype, tmp_path):
    """bin/trace_run as a user calls it, on a Pekodra folder: steps on standard input, logits as files."""
    config = CONFIGS["alone"]
    folder, w = make_folder(config, seed=27, folder=tmp_path / "m")
    reqs = {f"q{i}": p for i, p in enumerate(prompts(config["vocab"], [50, 3, 71, 20, 130], seed=7))}
    steps, peak = traces.mixed(reqs, {rid: max(1, len(t) - 5) for rid, t in reqs.items()}, seed=1, live=4, page=64)
    out = tmp_path / "out"
    proc = subprocess.run(
        [sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out),
         "--max-tokens", str(peak)],
        input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == [f"done {s['step']}" for s in steps]
    want = {rid: oracle(config, w, t) for rid, t in reqs.items()}
    at = {rid: 0 for rid in reqs}
    for s in steps:
        wanted = sum(len(e["want"]) for e in s["entries"])
        if not wanted:
            continue
        data = np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(wanted, config["vocab"])
        row = 0
        for e in s["entries"]:
            for k in e["want"]:
                logits, least = want[e["id"]]
                p = at[e["id"]] + k
                if least[p] >= CLOSE_CALL[dtype]:
                    assert np.abs(data[row] - logits[p]).max() <= TOL[dtype] * np.abs(logits).max(), (s["step"], e["id"], k)
                row += 1
            at[e["id"]] += len(e["tokens"])


# --------------------------------------------------------------------------- the kernels' new options one by one


def _close(got, want, tol, what):
    got, want = got.double().cpu(), want.double().cpu()
    err = float((got - want).abs().max() / max(1e-30, float(want.abs().max())))
    assert err <= tol, f"{what}: {err:.3g}"


@pytest.mark.gpu
@pytest.mark.parametrize("n,c", [(9, 20), (300, 52), (7, 50), (1, 1), (33, 1024), (5, 2048), (3, 3080), (2, 8192), (2, 8200), (40, 136)])
def test_two_norms_in_one_pass_and_rounded_rows(n, c):
    from akas_b200.ops import cuda, reference

    cuda.require(["elementwise"])
    g = torch.Generator().manual_seed(n * 1000 + c)
    x = (torch.randn(n, c, generator=g) * 3).cuda()
    w1, w2 = torch.randn(c, generator=g).cuda(), torch.randn(c, generator=g).cuda()
    for centered in (True, False):
        for dtype, tol in ((torch.float32, 2e-6), (torch.bfloat16, 8e-3)):
            for got, want in zip(cuda.rmsnorm_pair(x, w1, w2, 1e-3, centered, dtype), reference.rmsnorm_pair(x, w1, w2, 1e-3, centered, dtype)):
                _close(got, want, tol, f"two norms, {dtype}")
            wide = torch.full((n, 2 * c), 7.0, dtype=dtype, device="cuda")
            cuda.round_rows(x, wide[:, c:])
            assert torch.equal(wide[:, c:], x.to(dtype)) and bool((wide[:, :c] == 7.0).all())
            cuda.round_rows(x, wide[:, :c])
            assert torch.equal(wide, torch.cat([x, x], dim=1).to(dtype))


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,dims,page", [(6, 2, 24, 16, 16, 8), (3, 1, 20, 28, 6, 4), (5, 5, 12, 10, 0, 16),
                                                              (8, 2, 64, 48, 64, 64), (2, 1, 128, 64, 32, 64), (1, 1, 6, 2, 2, 8)])
def test_unit_heads_behind_the_rotation_kernel(heads, kv_heads, dim, vdim, dims, page, dtype):
    from akas_b200.ops import cuda, reference

    cuda.require(["attention_general"])
    rot = dict(base=300.0, dims=dims, scaling=BLEND)
    q, k, v, table, seq, pos, pages = _unit_case(heads, kv_heads, dim, vdim, rot, page)
    q, k, v = (x.to(dtype) for x in (q, k, v))
    tables = {}
    if dims:
        freq, amp = plain.rates(rot)
        cos, sin = reference.rope_tables(pos, torch.tensor(freq, dtype=torch.float64), amp)
    results = []
    for ops, device in ((reference, "cpu"), (cuda, "cuda")):
        if dims:
            tables = dict(cos=cos.to(device), sin=sin.to(device))
        for interleaved in (False, True):
            pools = [torch.zeros(pages, kv_heads, page, width, dtype=dtype, device=device) for width in (dim, vdim)]
            out = ops.qk_norm_store(q.to(device), k.to(device), v.to(device), heads, kv_heads, dim, vdim, None, None, 0.0, *pools,
                                    table.to(device), seq.to(device), pos.to(device), page, interleaved=interleaved, unit_eps=1e-4, **tables)
            results.append((out, *pools))
    tol = 2e-6 if dtype == torch.float32 else 8e-3
    for want, got in zip(results[:2], results[2:]):
        for a, b, what in zip(got, want, ("queries", "keys", "values")):
            _close(a, b, tol, what)
    # the same kernel with a weighted norm in front of the rotation, and with biases on float32 products
    g = torch.Generator().manual_seed(1)
    weights = [torch.rand(dim, generator=g) + 0.5 for _ in range(2)]
    biases = [torch.randn(width, generator=g) for width in (heads * dim, kv_heads * dim, kv_heads * vdim)]
    for weighted in (False, True):
        pair = []
        for ops, device in ((reference, "cpu"), (cuda, "cuda")):
            if dims:
                tables = dict(cos=cos.to(device), sin=sin.to(device))
            pools = [torch.zeros(pages, kv_heads, page, width, dtype=dtype, device=device) for width in (dim, vdim)]
            w = [x.to(device) if weighted else None for x in weights]
            out = ops.qk_norm_store(q.float().to(device), k.float().to(device), v.float().to(device), heads, kv_heads, dim, vdim, *w, 1e-4,
                                    *pools, table.to(device), seq.to(device), pos.to(device), page, **tables,
                                    **dict(zip(("q_bias", "k_bias", "v_bias"), (b.to(device) for b in biases))))
            pair.append((out, *pools))
        for a, b, what in zip(pair[1], pair[0], ("queries", "keys", "values")):
            _close(a, b, tol, f"{what}, biases, weights {weighted}")
    want = plain.rms(plain.rotate(q.double().reshape(-1, heads, dim), rot) if dims else q.double().reshape(-1, heads, dim), 1e-4)
    _close(results[2][0].reshape(-1, heads, dim), want, tol, "queries against the equations")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,dims,page", [(6, 2, 16, 12, 8), (4, 1, 32, 32, 16), (8, 2, 64, 32, 64), (5, 5, 64, 64, 64),
                                                         (2, 1, 128, 64, 64), (3, 3, 48, 0, 8), (2, 1, 256, 16, 32)])
def test_unit_heads_from_the_stacked_product(heads, kv_heads, dim, dims, page, dtype):
    """The kernel between the stacked q, k, v product and plain attention, and (head size 64, bfloat16) the decode kernel
    that does it on its way: heads divided by their root mean square behind the rotation."""
    from akas_b200.ops import cuda, reference

    cuda.require(["rope", "attention"] + (["attention_decode"] if dtype == torch.bfloat16 else []))
    rot = dict(base=300.0, dims=dims, scaling=BLEND)
    q, k, v, table, seq, pos, pages = _unit_case(heads, kv_heads, dim, dim, rot, page)
    qkv = torch.cat([q, k, v], dim=1).to(dtype)
    tables = (None, None)
    if dims:
        freq, amp = plain.rates(rot)
        tables = reference.rope_tables(pos, torch.tensor(freq, dtype=torch.float64), amp)
    results = []
    for ops, device in ((reference, "cpu"), (cuda, "cuda")):
        pools = [torch.zeros(pages, kv_heads, page, dim, dtype=dtype, device=device) for _ in range(2)]
        at = [t.to(device) if t is not None else None for t in tables]
        out = ops.qk_norm_rope_store(qkv.clone().to(device), heads, kv_heads, dim, None, None, 1e-4, False, *at, *pools, table.to(device),
                                     seq.to(device), pos.to(device), page, unit=True)
        results.append((out, *pools))
    tol = 2e-6 if dtype == torch.float32 else 8e-3
    for a, b, what in zip(results[1], results[0], ("queries", "keys", "values")):
        _close(a, b, tol, what)
    turned = qkv[:, : heads * dim].double().reshape(-1, heads, dim)
    _close(results[1][0].reshape(-1, heads, dim), plain.rms(plain.rotate(turned, rot) if dims else turned, 1e-4), tol, "against the equations")
    if dtype == torch.bfloat16 and dim == 64:
        # the last token decoded: its page row is not there yet
        class Ctx:
            max_context = 64
            query_lens = (1,)

        n = qkv.shape[0]
        want = reference.paged_attention(results[0][0][n - 1:], *results[0][1:], table, seq[n - 1:], pos[n - 1:], 0.2, 21, page)
        pools = [p.clone() for p in results[1][1:]]
        where = int(table[0, (n - 1) // page]), (n - 1) % page
        for p in pools:
            p[where[0], :, where[1]] = 0.0
        one = [t[n - 1:].cuda().contiguous() if t is not None else None for t in tables]
        got = cuda.qkv_decode_attention(qkv[n - 1:].cuda().contiguous(), heads, kv_heads, dim, None, None, 1e-4, False, *one, *pools, table.cuda(),
                                        seq[n - 1:].cuda(), pos[n - 1:].cuda(), 0.2, 21, page, Ctx, unit=True)
        assert got is not None
        _close(got, want, 1.5e-2, "decode attention from the product")
        _close(pools[0], results[1][1], 8e-3, "the key written on the way")
        assert torch.equal(pools[1], results[1][2])


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts,top,c,f", [(6, 2, 80, 24), (5, 1, 48, 16), (3, 3, 52, 20), (16, 2, 160, 136), (64, 6, 1104, 24),
                                             (1, 1, 24, 8), (4, 2, 264, 520)])
def test_ungated_experts(experts, top, c, f, dtype):
    from akas_b200.ops import cuda, reference

    cuda.require(["moe"] + (["moe_grouped"] if dtype == torch.bfloat16 else []))
    g = torch.Generator().manual_seed(experts * 100 + c)
    n = 75
    h = torch.randn(n, c + 8, generator=g).to(dtype).cuda()[:, :c]
    w_router = (torch.randn(experts, c, generator=g) * (3.0 / c ** 0.5)).cuda()
    want = reference.moe_route(h, w_router, None, 1, 1, top)
    got = cuda.moe_route(h, w_router, None, 1, 1, top)
    same = (got[0] == want[0]).all(dim=1)  # a choice may differ where two logits are within rounding of each other
    assert same.float().mean() > 0.9
    _close(got[1][same], want[1][same], 1e-4, "weights")
    chosen, weights = want
    best, at = torch.topk(h.float() @ w_router.T, top, dim=-1)
    held = (at == chosen.long()).all(dim=1)
    _close(weights[held], torch.softmax(best, dim=-1)[held], 1e-4, "the softmax over the chosen alone")
    # logits so far apart that all scores but one vanish: the choice still goes by the logits
    far = cuda.moe_route(h, w_router * 300.0, None, 1, 1, top)
    assert (far[0] == torch.topk(h.float() @ (w_router * 300.0).T, top, dim=-1).indices).all(dim=1).float().mean() > 0.9
    w_up = (torch.randn(experts, f, c, generator=g) * c ** -0.5).to(dtype).cuda()
    w_down = (torch.randn(experts, c, f, generator=g) * f ** -0.5).to(dtype).cuda()
    shared = torch.randn(n, c, generator=g).cuda()
    stream, beside = torch.randn(n, c, generator=g).cuda(), torch.randn(n, c, generator=g).cuda()
    tol = 2e-5 if dtype == torch.float32 else 1.5e-2
    for rows in (n, 5):  # 75 tokens: the grouped product in bfloat16 where it takes the sizes; 5: token by token
        sl = slice(0, rows)
        for activation in ("relu2", "gelu_tanh", "silu"):
            for sh in (None, (shared[sl].contiguous(), None)):
                ref = reference.moe_experts(h[sl], w_up, w_down, chosen[sl], weights[sl], shared=sh, activation=activation)
                out = cuda.moe_experts(h[sl], w_up, w_down, chosen[sl], weights[sl], shared=sh, activation=activation)
                _close(out, ref, tol, f"{activation}, {rows} tokens")
        x = stream[sl].clone()
        out = cuda.moe_experts(h[sl], w_up, w_down, chosen[sl], weights[sl], update=(x, beside[sl].contiguous(), None, None, 1.0),
                               shared=(shared[sl].contiguous(), None), activation="relu2")
        assert out is x
        ref = reference.moe_experts(h[sl], w_up, w_down, chosen[sl], weights[sl], shared=(shared[sl], None), activation="relu2")
        _close(out, stream[sl] + beside[sl] + ref, tol, "into the stream")
    # the statement itself, token by token in float64
    t = 3
    direct = torch.zeros(c, dtype=torch.float64)
    for e, wgt in zip(chosen[t].tolist(), weights[t].double().cpu()):
        direct += wgt * (w_down[e].double().cpu() @ (torch.relu(w_up[e].double().cpu() @ h[t].double().cpu()) ** 2))
    bare = cuda.moe_experts(h, w_up, w_down, chosen, weights, activation="relu2")
    _close(bare[t], direct, 5e-5 if dtype == torch.float32 else 3e-2, "the weighted sum of experts")
    if dtype == torch.bfloat16:
        assert cuda.moe_grouped_status() == 0


@pytest.mark.gpu
@pytest.mark.parametrize("m,k,f", [(1, 128, 48), (3, 64, 16), (8, 2048, 1024), (9, 1024, 72), (16, 512, 200), (16, 2048, 40)])
def test_a_norm_in_front_of_the_gated_product(m, k, f):
    """RMSNorm on the skinny product's way in, biases and gelu in its read-out, against the steps one by one."""
    from akas_b200.ops import cuda, reference

    cuda.require(cuda.libraries_for(torch.bfloat16, ()))
    g = torch.Generator().manual_seed(m * 7 + f)
    h = (torch.randn(m + 2, k, generator=g) * 3).cuda()
    nw = (torch.randn(k, generator=g) * 0.3).cuda()
    w = (torch.randn(2 * f, k, generator=g) * k ** -0.5).to(torch.bfloat16).cuda()
    bias = torch.randn(2 * f, generator=g).cuda()
    rows = (torch.arange(m, dtype=torch.int32) + 1).cuda()
    for picked in (None, rows):
        x = h[:m].contiguous() if picked is None else h
        for b in (None, bias):
            for activation in ("gelu_tanh", "silu"):
                got = cuda.norm_linear_gated(x, nw, 1e-5, True, w, f, b, activation, picked)
                assert got is not None
                want = reference.linear_gated(reference.rmsnorm(x, nw, 1e-5, True, torch.bfloat16, picked), w, f, b, activation)
                _close(got, want, 1.5e-2, f"{activation} behind a norm")
    assert cuda.skinny_status() == 0
    assert cuda.norm_linear_gated(h[:1].repeat(17, 1), nw, 1e-5, True, w, f, bias, "silu") is None  # more tokens than it takes


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layer_widths_of_a_real_model(dtype, tmp_path):
    """Widths at which every product, the attention and the grouped experts run on their tensor-core kernels (a width of
    1,024, heads of 64 and 128, sixteen experts of 768), a prompt of 700 tokens in one step, in portions beside another
    request, and its last tokens decoded: against the plain model."""
    from akas_b200.engine.batch import StepEntry

    wide = attn(16, 4, 64, 64, 300, 0.25, 500000.0, 64, dict(factor=8.0, original=4096, fast=32.0, slow=1.0))
    long = attn(8, 2, 128, 128, 513, 0.15, 1000000.0, 64, dict(factor=4.0, original=256, fast=16.0, slow=2.0))
    # (only the last layer routes: a choice that falls the other way then moves its own position and no later one)
    config = model(1024, 2048, [layer(wide, dense(3072)), layer(long, dense(1024)), layer(wide, None), layer(long, moe(768, 16, 3, shared=1024))],
                   loop=(1, 3, 2), eps=1e-6, logit_scale=1024 ** -0.5)
    folder, w = make_folder(config, seed=5, folder=tmp_path / "m", std=0.02)
    toks, other = prompts(config["vocab"], [700, 150], seed=3)
    logits, least = oracle(config, w, toks)
    held = least >= {"float32": 1e-3, "bfloat16": 0.05}[dtype]
    rows = list(range(0, 700, 37)) + list(range(690, 700))
    tol = TOL[dtype]

    def check(got, at, what):
        keep = [i for i, p in enumerate(at) if held[p]]
        assert len(keep) > len(at) // 2
        err = np.abs(got[keep] - logits[np.asarray(at)[keep]]).max() / np.abs(logits).max()
        assert err <= tol, f"{what}: {err:.3g}"

    runner = runner_for(folder, dtype, "cuda:0", 64, 1024, None, max_requests=2, context=768)
    check(runner.step([StepEntry("a", toks, tuple(rows))]).float().cpu().numpy(), rows, "one step")
    runner.release("a")
    at, got, places = 0, [], []
    for k, (count, beside) in enumerate(((300, 100), (2, 0), (130, 50), (258, 0))):
        entries = [StepEntry("a", toks[at:at + count], tuple(range(count)))]
        if beside:
            entries.append(StepEntry("b", other[:beside] if k == 0 else other[100:150], ()))
        got.append(runner.step(entries).float().cpu().numpy())
        places += list(range(at, at + count))
        at += count
    for p in range(at, 700):
        got.append(runner.step([StepEntry("b", (5,), ()), StepEntry("a", toks[p:p + 1], (0,))]).float().cpu().numpy())
        places.append(p)
    check(np.concatenate(got), places, "portions beside another request, then single tokens")
