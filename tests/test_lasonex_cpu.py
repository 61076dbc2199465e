"""The Lasonex design through the package's own configuration, loader, cache, state and step function on the CPU, with every CUDA
kernel replaced by its plain reference (the `reference_kernels` fixture), against the plain implementation of
tests/plain_lasonex.py. This checks the host side: names and shapes, the order of the parts, heads of two maps and their padding, what
every kind of layer keeps per sequence, what stays pending between layers, pages given back as a window passes. The kernels themselves
are checked on a GPU."""
import math

import pytest
import torch

from tests import plain_lasonex as plain
from tests.helpers import max_err, random_tokens
from tests.helpers_lasonex import (CONFIGS, LAS_FAST, LAS_ODD, LAS_ONES, STRETCH, attention, config, dense, layer, make_model_dir, moe, retention)


def build(cfg, tmp_path, seed=0):
    from qwenforge_b200.engine import Model
    folder, weights = make_model_dir(cfg, seed, tmp_path)
    return Model.from_dir(folder, "float32", "cpu"), weights, folder


def run(model, cache, tokens, cuts):
    slot, at, got = cache.open(), 0, []
    for size in list(cuts) + [1] * (len(tokens) - sum(cuts)):
        got.append(model.step(cache, [(slot, tokens[at:at + size])], want=[list(range(size))]))
        at += size
    cache.close(slot)
    return torch.cat(got)


def test_configuration_names_every_tensor():
    from qwenforge_b200.config import LasonexConfig, config_from_dict, preset_config
    from qwenforge_b200.engine import Model
    for cfg in CONFIGS.values():
        cfg_obj = config_from_dict(cfg)
        assert isinstance(cfg_obj, LasonexConfig)
        spec = cfg_obj.model_spec()
        wanted = {t.name: tuple(t.shape) for t in Model.tensor_specs_of(spec)}
        assert wanted == plain.tensor_shapes(cfg)
        assert config_from_dict(cfg_obj.to_dict()).model_spec() == spec
        assert [e.layer for e in spec.schedule] == list(range(len(cfg["layers"])))
    assert config_from_dict(LAS_ODD).model_spec().ignored_tensors == ("l1.norm2",)   # a layer without a feed-forward has no second norm
    for name in ("lasonex-tiny", "lasonex-0.5b", "lasonex-3b"):
        assert preset_config(name).model_spec().architecture == "Lasonex"
    bad = lambda *layers: config(50, 16, 1e-6, 1.0, list(layers))
    with pytest.raises(ValueError, match="not supported"):
        config_from_dict(bad(dict(type="other", mixer={}, mlp=None)))
    with pytest.raises(ValueError, match="top"):
        config_from_dict(bad(layer(retention(1, 8, 8, 8), moe(2, 3, 4))))
    with pytest.raises(ValueError, match="groups"):
        config_from_dict(bad(layer(retention(1, 8, 8, 8), moe(6, 3, 4, groups=(3, 1)))))
    with pytest.raises(ValueError, match="decay"):
        config_from_dict(bad(layer(retention(3, 8, 8, 8, decay=[0.5]), None)))
    with pytest.raises(ValueError, match="kv_heads"):
        config_from_dict(bad(layer(attention(3, 2, 8, 8, 8, 8), None)))
    with pytest.raises(ValueError, match="dims"):
        config_from_dict(bad(layer(attention(2, 2, 8, 8, 8, 10), None)))
    with pytest.raises(ValueError, match="scale"):
        config_from_dict({k: v for k, v in LAS_ONES.items() if k != "embedding"} | {"embedding": {}})


def test_what_a_layer_keeps(reference_kernels, tmp_path):
    """Keys of both maps side by side in one cached head, filled up to a size that the tensor-core kernels have; one state per head."""
    from qwenforge_b200.cache import KvNeed, StateNeed
    model, _, _ = build(LAS_ODD, tmp_path)
    needs = model.cache_needs()
    assert needs[0] == KvNeed(2, 32, 7) and needs[2] == KvNeed(3, 32, 90) and needs[4] == KvNeed(2, 32, 33)
    assert needs[1] == StateNeed((3 * 10 * 6,)) and needs[3] == StateNeed((2 * 6 * 22,))
    fast, _, _ = build(LAS_FAST, tmp_path / "fast")
    assert [n.head_dim for n in fast.cache_needs() if isinstance(n, KvNeed)] == [64, 32, 96, 128]


@pytest.mark.parametrize("name", list(CONFIGS))
def test_every_cut_agrees_with_the_plain_implementation(reference_kernels, name, tmp_path):
    cfg = CONFIGS[name]
    model, weights, _ = build(cfg, tmp_path, seed=1)
    tokens = random_tokens(cfg["vocab"], 80, 3)
    want = plain.forward_logits(cfg, weights, tokens)
    cache = model.new_cache(512, 2)
    for cuts in ([80], [37, 2, 20], [64, 2], [1, 65]) + (([],) if name != "fast" else ()):
        got = run(model, cache, tokens, cuts)
        assert max_err(got, want) < 2e-4, (name, cuts)
    assert all(g.pages.n_free == g.pages.n_pages for g in cache.kv_groups)


def test_pages_leave_as_the_window_passes_and_slots_come_back_clean(reference_kernels, tmp_path):
    cfg = config(40, 16, 1e-5, 2.0, [layer(attention(2, 1, 4, 8, 10, 4), None), layer(retention(2, 4, 6, 4), dense(8))])
    model, weights, _ = build(cfg, tmp_path, seed=5)
    cache = model.new_cache(64 * 6, 2)
    windowed = cache.kv_groups[0]
    tokens = random_tokens(40, 200, 4)
    want = plain.forward_logits(cfg, weights, tokens)
    slot = cache.open()
    got = [model.step(cache, [(slot, tokens[:70])], want=[list(range(70))])]
    for t in range(70, 200):
        got.append(model.step(cache, [(slot, [tokens[t]])]))
        assert windowed.pages_held(slot) <= 2
    assert max_err(torch.cat(got), want) < 2e-4
    cache.close(slot)
    # the slot and its state rows again, for another sequence: nothing of the first one is left
    other = random_tokens(40, 30, 8)
    assert max_err(run(model, cache, other, [30]), plain.forward_logits(cfg, weights, other)) < 2e-4
    assert max_err(run(model, cache, other, [12]), plain.forward_logits(cfg, weights, other)) < 2e-4


def test_unequal_batches_against_each_request_alone(reference_kernels, tmp_path):
    model, weights, _ = build(LAS_ODD, tmp_path, seed=2)
    cache = model.new_cache(64 * 8, 3)
    seqs = [random_tokens(LAS_ODD["vocab"], n, 30 + n) for n in (40, 3, 17)]
    want = [plain.forward_logits(LAS_ODD, weights, s) for s in seqs]
    for _ in range(2):
        slots = [cache.open() for _ in seqs]
        heads = [max(1, len(s) - 5) for s in seqs]
        logits = model.step(cache, [(slots[i], seqs[i][:heads[i]]) for i in range(3)], want=[list(range(h)) for h in heads])
        got, o = [[] for _ in seqs], 0
        for i, h in enumerate(heads):
            got[i].append(logits[o:o + h])
            o += h
        fed = list(heads)
        live = [i for i in range(3) if fed[i] < len(seqs[i])]
        while live:
            logits = model.step(cache, [(slots[i], [seqs[i][fed[i]]]) for i in live])
            for row, i in enumerate(live):
                got[i].append(logits[row:row + 1])
                fed[i] += 1
            live = [i for i in live if fed[i] < len(seqs[i])]
        for i in range(3):
            cache.close(slots[i])
            assert max_err(torch.cat(got[i]), want[i]) < 2e-4


def test_the_stream_after_every_layer(reference_kernels, tmp_path):
    """What stays pending (the mixer's output and the experts' unsummed rows) is worth what the plain layer adds."""
    model, weights, _ = build(LAS_ODD, tmp_path)
    tokens = random_tokens(LAS_ODD["vocab"], 30, 1)
    seen = {}
    model.observer = lambda i, hidden, delta: seen.__setitem__(i, (hidden if delta is None else hidden + delta.float()).clone())
    run(model, model.new_cache(256, 2), tokens, [30])
    streams = []
    plain.forward(LAS_ODD, weights, tokens, streams)
    assert max_err(seen[0], weights["embed"][tokens] * 3.0) < 1e-6
    for i, stream in enumerate(streams):
        assert max_err(seen[i + 1], stream) < 2e-4, f"after layer {i}"


def test_the_plain_mechanisms_on_made_cases():
    """The router, the frequencies, the combination of two maps and the recurrence on numbers chosen by hand."""
    mlp = moe(6, 2, 4, groups=(3, 1))
    weights = {"r.router": torch.eye(6, 6)}
    z = torch.tensor([[1.0, 0.9, 1.1, -5.0, 0.8, 0.7]], dtype=torch.float64)
    chosen, weight, margin = plain.router(weights, "r.", mlp, z)
    # the second group holds the largest score, so both of its experts are chosen although one is the worst of all
    assert sorted(chosen.tolist()[0]) == [2, 3] and abs(float(weight.sum()) - 1.0) < 1e-12
    assert abs(float(weight[0, 0] / weight[0, 1]) - math.exp(6.1)) < 1e-6 and abs(float(margin[0]) - 0.1) < 1e-9
    freq, amplitude = plain.frequencies(dict(dims=8, base=100.0, scaling=dict(factor=4.0, original=64, fast=8.0, slow=0.5)))
    # dim(8) = 8 ln(64 / (16 pi)) / (2 ln 100) = 0.21 -> lo 0; dim(0.5) = 2.62 -> hi 3: pairs 0 .. 3 from whole to a quarter
    assert max(abs(a - b) for a, b in zip(freq, [1.0, 100 ** -0.25 * (1 - 0.75 / 3), 0.1 * 0.5, 100 ** -0.75 / 4])) < 1e-12
    assert abs(amplitude - (0.1 * math.log(4.0) + 1.0)) < 1e-12
    o = plain.combine_maps(torch.tensor([3.0, 1.0], dtype=torch.float64), torch.tensor([0.0, 10.0], dtype=torch.float64), 0.5, 0.2, 0.0)
    assert max_err(o, 0.8 * torch.tensor([3.0, -4.0], dtype=torch.float64) / math.sqrt(12.5)) < 1e-12
    ones = torch.ones(3, 1, dtype=torch.float64)
    assert plain.retain(ones, ones, torch.tensor([[1.0], [0.0], [2.0]], dtype=torch.float64), 0.5).flatten().tolist() == [1.0, 0.5, 2.25]


def test_stretched_frequencies_of_the_position_part():
    from qwenforge_b200.config import PartSpec
    from qwenforge_b200.parts import build_part
    for dims, base in ((8, 100.0), (20, 50000.0)):
        rot = dict(dims=dims, base=base, scaling=STRETCH)
        part = build_part("position", PartSpec("rotary_half", {"head_dim": 24, "rotary_dim": dims, "theta": base, "precise": True, "scaling": STRETCH}))
        part.bind({}, torch.float32, "cpu")
        freq, amplitude = plain.frequencies(rot)
        assert max_err(part.inv_freq, torch.tensor(freq, dtype=torch.float64)) < 1e-7 and abs(part.amplitude - amplitude) < 1e-12


def test_generation_loop_on_the_cpu(reference_kernels, tmp_path):
    from qwenforge_b200.engine import StudentEngine
    folder, weights = make_model_dir(LAS_ONES, 6, tmp_path)
    prompts = [random_tokens(LAS_ONES["vocab"], n, n) for n in (5, 20, 1)]
    want = [plain.greedy_generate(LAS_ONES, weights, p, 6) for p in prompts]
    engine = StudentEngine(str(folder), device="cpu", dtype="float32", cuda_graphs=False)
    assert engine.generate_ids(prompts, max_new_tokens=6, batch_size=2, ignore_eos=True) == want
