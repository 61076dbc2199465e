"""The Dapupel design through the package's own configuration, loader, cache, state and step function on the CPU, with every CUDA
kernel replaced by its plain reference (the `reference_kernels` fixture), against the plain implementation of
tests/plain_dapupel.py. This checks the host side: names and shapes, the streams and what is pending for them, what every
kind of layer and every sublayer's filter keeps per sequence, padded rows of the latent cache, pages given back as a window passes.
The kernels themselves are checked on a GPU."""
import math

import pytest
import torch

from tests import plain_dapupel as plain
from tests.helpers import max_err, random_tokens
from tests.helpers_dapupel import (CONFIGS, DAP_FAST, DAP_ODD, DAP_ONES, attention, config, delta, latent, layer, make_model_dir, moe)


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
    from qwenforge_b200.config import DapupelConfig, config_from_dict
    from qwenforge_b200.engine import Model
    for cfg in CONFIGS.values():
        cfg_obj = config_from_dict(cfg)
        assert isinstance(cfg_obj, DapupelConfig)
        spec = cfg_obj.model_spec()
        wanted = {t.name: tuple(t.shape) for t in Model.tensor_specs_of(spec)}
        shapes = plain.tensor_shapes(cfg)
        assert set(wanted) == set(shapes)
        assert all(len(wanted[n]) == len(shapes[n]) and all(a in (-1, b) for a, b in zip(wanted[n], shapes[n])) for n in shapes)
        assert config_from_dict(cfg_obj.to_dict()).model_spec() == spec
        assert [e.layer for e in spec.schedule] == list(range(len(cfg["layers"])))
    # what belongs to a feed-forward that a layer does not have may stand in a file and is not read
    spec = config_from_dict(DAP_ODD).model_spec()
    assert {"l2.norm2", "l2.norm2.alpha", "l2.hc2.mix", "l2.canon2"} <= set(spec.ignored_tensors)
    for mixer, mlp, match in ((("other", {}), None, "not supported"), (delta(3, 2, 8, 8), None, "kv_heads"),
                              (attention(2, 2, 8, 4), moe(2, 3, 4), "top"), (attention(2, 2, 8, 0), None, "size"),
                              (latent(2, 8, 3, 8, 8, 8), None, "rot"), (attention(2, 2, 8, 4), dict(kind="dense", ff=4), "dense")):
        with pytest.raises(ValueError, match=match):
            config_from_dict(config(50, 16, 2, 4, 1e-6, [layer(mixer, mlp)]))
    wrong = attention(2, 2, 8, 4)
    wrong[1]["vdim"] = 6
    with pytest.raises(ValueError, match="vdim"):
        config_from_dict(config(50, 16, 2, 4, 1e-6, [layer(wrong, None)]))
    with pytest.raises(ValueError, match="streams"):
        config_from_dict({k: v for k, v in DAP_ONES.items() if k != "streams"})


def test_what_a_layer_keeps(reference_kernels, tmp_path):
    from qwenforge_b200.cache import BundleNeed, KvNeed, StateNeed
    model, _, _ = build(DAP_ODD, tmp_path)
    needs = [dict(n.items) for n in model.cache_needs()]
    filter_ = StateNeed((2 * 44,))
    assert all(n["mixer_input"] == filter_ for n in needs)
    assert [("feed_forward_input" in n) for n in needs] == [True, True, False, True, True]
    assert needs[0]["mixer"] == StateNeed((420 + 104,))                       # six states of 10 x 7, one row of 30 + 30 + 42 inputs, filled up
    window = dict(needs[1]["mixer"].items)
    assert window["kv"] == KvNeed(2, 6, 9, planes=1) and window["conv"] == StateNeed((2 * (24 + 12),))
    assert needs[2]["mixer"] == KvNeed(1, 32, 0, planes=1)                    # 14 + 6 numbers, filled up to the kernels' smallest rows
    assert needs[3]["mixer"] == KvNeed(1, 32, 0, planes=1)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_every_cut_agrees_with_the_plain_implementation(reference_kernels, name, tmp_path):
    cfg = CONFIGS[name]
    model, weights, _ = build(cfg, tmp_path, seed=1)
    tokens = random_tokens(cfg["vocab"], 90, 3)
    want = plain.forward_logits(cfg, weights, tokens)
    cache = model.new_cache(512, 2)
    for cuts in ([90], [37, 2, 20], [], [64, 2], [1, 65]):
        got = run(model, cache, tokens, cuts)
        assert max_err(got, want) < 2e-4, (name, cuts)
    assert all(g.pages.n_free == g.pages.n_pages for g in cache.kv_groups)


def test_pages_leave_as_the_window_passes_and_slots_come_back_clean(reference_kernels, tmp_path):
    cfg = config(40, 16, 2, 4, 1e-5, [layer(attention(2, 1, 8, 10), None), layer(delta(2, 2, 4, 4, ranks=(2, 2)), moe(2, 1, 8)),
                                      layer(latent(2, 4, 2, 4, 6, 5), None)])
    model, weights, _ = build(cfg, tmp_path, seed=5)
    cache = model.new_cache(64 * 6, 2)
    windowed = [g for g in cache.kv_groups if g.need.window == 10][0]
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
    for cuts in ([30], [12], [2]):
        assert max_err(run(model, cache, other, cuts), plain.forward_logits(cfg, weights, other)) < 2e-4


def test_unequal_batches_against_each_request_alone(reference_kernels, tmp_path):
    model, weights, _ = build(DAP_ODD, tmp_path, seed=2)
    cache = model.new_cache(64 * 8, 3)
    seqs = [random_tokens(DAP_ODD["vocab"], n, 30 + n) for n in (40, 3, 17)]
    want = [plain.forward_logits(DAP_ODD, weights, s) for s in seqs]
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


def test_stretched_frequencies_of_the_rotation():
    """The frequencies and the factor on cosine and sine against the plain implementation, where the ramp lies inside, at both ends
    and where it is empty."""
    from qwenforge_b200.config import PartSpec
    from qwenforge_b200.parts import build_part
    for dims, base, scaling in ((32, 10000.0, (4.0, 256, 32.0, 1.0)), (16, 5e5, (8.0, 4096, 32.0, 1.0)), (8, 100.0, (2.0, 7, 64.0, 40.0)),
                                (2, 1e4, (4.0, 64, 8.0, 8.0))):
        named = dict(zip(("factor", "original", "fast", "slow"), scaling))
        part = build_part("position", PartSpec("rotary_interleaved", dict(head_dim=dims, theta=base, precise=True, scaling=named)))
        part.bind({}, torch.float32, "cpu")
        want, factor = plain.frequencies(dict(dims=dims, base=base, scaling=named))
        assert max_err(part.fused_rotary()[0].double() / want, torch.ones(dims // 2).double()) < 1e-6
        assert abs(part.amplitude - factor) < 1e-12 and abs(factor - (1 + 0.1 * math.log(scaling[0]))) < 1e-12


def test_the_ranks_of_the_low_rank_pairs_come_from_the_tensors(reference_kernels, tmp_path):
    model, _, _ = build(DAP_ODD, tmp_path)
    part = dict((s[0], s[4]) for s in model.blocks[0].sublayers)["mixer"]
    assert (part.rank, part.gate_rank) == (3, 5)


def test_another_norm_among_several_streams(reference_kernels, tmp_path):
    """The arrangement with a norm that sums over its row (it reads u as a row of its own, and the filter runs behind it) is the
    arrangement with the norm applied inside: checked by the same Dynamic Tanh with its elementwise form hidden."""
    cfg = DAP_ODD
    model, weights, _ = build(cfg, tmp_path, seed=3)
    tokens = random_tokens(cfg["vocab"], 40, 3)
    want = plain.forward_logits(cfg, weights, tokens)

    class Hidden:
        def __init__(self, norm):
            self.norm = norm

        def forward(self, hidden, delta):
            return self.norm.forward(hidden, delta)

        def fused_rms(self):
            return None

        def __getattr__(self, name):
            if name == "elementwise":
                raise AttributeError(name)
            return getattr(self.norm, name)

    for block in model.blocks:
        block.sublayers = [(name, streams, Hidden(norm), filter_, sub) for name, streams, norm, filter_, sub in block.sublayers]
    model.final_norm = Hidden(model.final_norm)
    assert max_err(run(model, model.new_cache(256, 2), tokens, [21, 2]), want) < 2e-4


def test_generation_loop_on_the_cpu(reference_kernels, tmp_path):
    from qwenforge_b200.engine import StudentEngine
    folder, weights = make_model_dir(DAP_ONES, 6, tmp_path)
    prompts = [random_tokens(DAP_ONES["vocab"], n, n) for n in (5, 20, 1)]
    want = [plain.greedy_generate(DAP_ONES, weights, p, 6) for p in prompts]
    engine = StudentEngine(str(folder), device="cpu", dtype="float32", cuda_graphs=False)
    assert engine.generate_ids(prompts, max_new_tokens=6, batch_size=2, ignore_eos=True) == want
