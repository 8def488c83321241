"""Lelutar without a GPU: configuration, tensor names, cache layout, the rotation table, and hand-worked anchors of the plain
implementation's functions."""
import copy
import json
import math

import pytest
import torch

import plain_lelutar as P
from lelutar_configs import LELUTAR_A, LELUTAR_B, LELUTAR_C, LELUTAR_D, LELUTAR_E, write_model

from ferrum_b200.config import registry
from ferrum_b200.config.lelutar import AttentionSpec, BigramSpec, LatentSpec, LelutarConfig
from ferrum_b200.errors import ConfigError, WeightsError

F64 = torch.float64


def test_config_reads_every_size_and_constant():
    c = LelutarConfig.from_dict(LELUTAR_A)
    assert (c.n_vocab, c.n_embd, c.norm_eps, c.n_layer, c.logit_scale, c.embedding_scale) == (197, 52, 1e-4, 7, 1.7, 3.5)
    assert c.bigram == BigramSpec(61, 31, 7)
    a, b, t = c.layers[0].mixer, c.layers[1].mixer, c.layers[2].mixer
    assert isinstance(a, AttentionSpec) and isinstance(b, LatentSpec) and isinstance(t, LatentSpec)
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.rot.base, a.rot.dims) == (6, 2, 10, 14, 0.45, 700.0, 6)
    s = a.rot.scaling
    assert (s.factor, s.original, s.fast, s.slow) == (3.0, 48.0, 9.0, 0.5)
    assert (b.heads, b.dim, b.vdim, b.kv_rank, b.q_rank, b.scale, b.rot_dim, b.rot) == (3, 7, 9, 11, 13, 0.6, 0, None)
    assert (t.heads, t.dim, t.vdim, t.kv_rank, t.q_rank, t.rot_dim, t.rot.dims) == (5, 6, 10, 18, 17, 4, 4)
    assert c.layers[6].mixer.rot.scaling is None
    assert c.layers[0].mlp.ff == 36 and c.layers[2].mlp is None
    m = c.layers[1].mlp
    assert (m.ff, m.experts, m.top, m.groups) == (20, 10, 3, (5, 3))
    assert [c.owner(i) for i in range(7)] == [0, 1, 2, 2, 1, 2, 6] and c.owners() == [0, 1, 2, 6]
    assert LelutarConfig.from_dict(LELUTAR_B).owner(0) == 3
    assert LelutarConfig.from_dict(LELUTAR_C).bigram is None
    d = LelutarConfig.from_dict(LELUTAR_D)
    assert d.layers[1].mixer.rot is None and d.layers[1].mlp.groups is None and d.logit_scale == -0.6


@pytest.mark.parametrize("edit,message", [
    (lambda d: d["layers"][0].update(type="mamba2"), "not a mixer"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda d: d["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=12), "rot.dims"),
    (lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0), "rot.scaling"),
    (lambda d: d["layers"][1]["mixer"].pop("q_rank"), "q_rank"),
    (lambda d: d["layers"][2]["mixer"].pop("rot_dim"), "rot_dim"),
    (lambda d: d["layers"][1]["mlp"]["router"].update(top=7), "groups"),
    (lambda d: d["layers"][1]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda d: d["layers"][1]["mlp"]["router"]["groups"].update(keep=6), "groups"),
    (lambda d: d["layers"][0]["mlp"].update(kind="gated"), "feed-forward"),
    (lambda d: d["layers"][4].update(weights_of=9), "weights_of"),
    (lambda d: d["layers"][4].update(weights_of=4), "weights_of"),
    (lambda d: d["layers"][4].update(weights_of=0), "differs"),
    (lambda d: d["layers"][2].update(weights_of=5), "circle"),
    (lambda d: d["embedding"]["bigram"].pop("mul_cur"), "mul_cur"),
    (lambda d: d["embedding"]["bigram"].update(buckets=0), "buckets"),
    (lambda d: d["norm"].update(eps=0.0), "eps"),
    (lambda d: d.pop("width"), "width"),
])
def test_config_refusals(edit, message):
    d = copy.deepcopy(LELUTAR_A)
    edit(d)
    with pytest.raises(ConfigError, match=message):
        LelutarConfig.from_dict(d)


def build(d, dtype=torch.float32, **kw):
    arch = registry.lookup("Lelutar")
    return arch.build(arch.read_config(d), dtype, "cpu", **kw), arch


@pytest.mark.parametrize("d", [LELUTAR_A, LELUTAR_B, LELUTAR_C, LELUTAR_D, LELUTAR_E])
def test_tensor_names_cover_the_model_and_the_file(tmp_path, d):
    """The map from file names hits every tensor that the parts declare, once; a written file loads, and a missing,
    an unknown and a misshapen tensor are named in one error."""
    from ferrum_b200.weights import load_weights
    from ferrum_b200.weights.safetensors_io import SafetensorsFile, write_safetensors
    model, arch = build(d)
    names = arch.hf_names(arch.read_config(d))
    assert sorted(names.values()) == sorted(model.weight_specs()) and len(set(names.values())) == len(names)
    folder = write_model(d, str(tmp_path / "m"), 3)
    cfg, w = P.load(folder)
    assert set(w) == set(names)
    assert ("bigram" in w) == ("bigram" in d["embedding"])
    for i, layer in enumerate(d["layers"]):
        own = layer.get("weights_of") is None
        assert any(n.startswith(f"l{i}.") for n in w) == own
        if own:
            assert w[f"l{i}.norm1.alpha"].shape == () and w[f"l{i}.norm1.b"].shape == (d["width"],)
            assert (f"l{i}.norm2" in w) == (layer["mlp"] is not None)
            assert (f"l{i}.mix.sink" in w) == (f"l{i}.mix.g" in w) == (layer["type"] != "attention") == (f"l{i}.mix.q.b" not in w)
    load_weights(model, folder, names, device="cpu")
    path = folder + "/model.safetensors"
    st = SafetensorsFile(path)
    tensors = {n: st.tensor(n).clone() for n in st.names()}
    tensors["l9.mix.q"] = tensors.pop("final.norm.alpha")
    tensors["head"] = tensors["head"][:, :-1].contiguous()
    write_safetensors(path, tensors, {"format": "pt"})
    with pytest.raises(WeightsError) as err:
        load_weights(build(d)[0], folder, names, device="cpu")
    assert all(s in str(err.value) for s in ("missing: final.norm.alpha", "unexpected: l9.mix.q", "head: shape"))


def test_layers_that_share_tensors_have_planes_of_their_own():
    from ferrum_b200.cache.storage import CacheLayout
    model, _ = build(LELUTAR_A)
    lay = CacheLayout(model)
    assert [r.block for r in model.schedule] == [0, 1, 2, 2, 1, 2, 3] and all(r.cache_of is None for r in model.schedule)
    assert lay.group_keys == [(2, 14, 0, 2), (1, 11, 0, 1), (1, 22, 0, 1), (3, 6, 0, 2)]
    assert lay.run_group == [0, 1, 2, 2, 1, 2, 3] and lay.run_plane == [0, 0, 0, 1, 1, 2, 0]
    assert lay.embedding_state == 0 and [(n.shape, n.dtype) for n in lay.state_needs] == [((1,), torch.int32)]
    lay = CacheLayout(build(LELUTAR_C)[0])
    assert lay.embedding_state is None and lay.state_needs == []


def test_the_embedding_state_is_per_slot_and_starts_from_zero():
    from ferrum_b200.cache import CacheStorage
    cache = CacheStorage(build(LELUTAR_A)[0], torch.float32, "cpu", page_size=8, max_tokens=64, max_requests=3)
    assert cache.embedding_state.shape == (3, 1) and cache.embedding_state.dtype == torch.int32
    cache.embedding_state.fill_(7)
    slot = cache.open()
    assert cache.embedding_state[slot].item() == 0 and (cache.embedding_state == 7).sum() == 2
    plain_cache = CacheStorage(build(LELUTAR_C)[0], torch.float32, "cpu", page_size=8, max_tokens=64, max_requests=3)
    assert plain_cache.embedding_state is None


def test_logit_scale_lives_in_the_last_norm(tmp_path):
    from ferrum_b200.weights import load_weights
    folder = write_model(LELUTAR_A, str(tmp_path / "m"), 3)
    model, arch = build(LELUTAR_A)
    load_weights(model, folder, arch.hf_names(arch.read_config(LELUTAR_A)), device="cpu")
    _, w = P.load(folder)
    assert torch.allclose(model.final_norm.w_weight.double(), w["final.norm"] * 1.7) and torch.allclose(model.final_norm.w_bias.double(), w["final.norm.b"] * 1.7)
    assert torch.allclose(model.blocks[0].norm1.w_weight.double(), w["l0.norm1"])


# --------------------------------------------------------------------------- the rotation
ROTS = [{"base": 700.0, "dims": 6, "scaling": {"factor": 3.0, "original": 48, "fast": 9.0, "slow": 0.5}},
        {"base": 10000.0, "dims": 64, "scaling": {"factor": 40.0, "original": 4096, "fast": 32.0, "slow": 1.0}},
        {"base": 50.0, "dims": 2, "scaling": {"factor": 2.0, "original": 16, "fast": 2.0, "slow": 1.0}},
        {"base": 1e6, "dims": 128, "scaling": {"factor": 1.0, "original": 100, "fast": 3.0, "slow": 3.0}},
        {"base": 300.0, "dims": 8, "scaling": {"factor": 8.0, "original": 4, "fast": 32.0, "slow": 8.0}}]


@pytest.mark.parametrize("rot", ROTS)
def test_yarn_table_against_the_plain_rule(rot):
    from ferrum_b200.parts import RotaryEmbedding
    from ferrum_b200.parts.rope import yarn
    s = rot["scaling"]
    f, mag = yarn(rot["dims"], rot["base"], s["factor"], s["original"], s["fast"], s["slow"])
    want, mult = P.frequencies(rot)
    assert f == pytest.approx(want, rel=1e-12) and mag == pytest.approx(mult)
    table = RotaryEmbedding(rot["dims"], rot["dims"], rot["base"], None, "adjacent", 5000, "cpu", frequencies=f, magnitude=mag)
    assert table.pairing == 0
    for p in (0, 1, 777, 4999):
        ang = torch.tensor(want, dtype=F64) * p
        assert torch.allclose(table.cos_sin[p].double(), torch.stack([torch.cos(ang), torch.sin(ang)], -1) * mult, atol=1e-6)


def test_plain_yarn_by_hand():
    """base 16, 4 dims: f = [1, 1/4].  Over 2 pi * 8 positions pair i makes 8 f_i turns: the pair that makes t turns is
    4 ln(8 / t) / (2 ln 16) = ln(8 / t) / ln 4."""
    rot = {"base": 16.0, "dims": 4, "scaling": {"factor": 2.0, "original": 16.0 * math.pi, "fast": 8.0, "slow": 0.5}}
    f, mult = P.frequencies(rot)             # fast: pair 0; slow: pair 2 -> ramp 0, 1/2
    assert f == pytest.approx([1.0, 0.25 * 0.5 * 0.5 + 0.25 * 0.5]) and mult == pytest.approx(1.0 + 0.1 * math.log(2.0))
    rot["scaling"].update(fast=1000.0, slow=8.0)        # fast: below 0 -> 0; slow: 0 -> the ramp is as good as a step behind pair 0
    assert P.frequencies(rot)[0] == pytest.approx([1.0, 0.125])
    rot["scaling"].update(fast=0.01, slow=0.001)        # the ramp starts behind every pair there is
    assert P.frequencies(rot)[0] == pytest.approx([1.0, 0.25])
    assert P.frequencies({"base": 16.0, "dims": 4}) == ([1.0, 0.25], 1.0)


def test_plain_rotation_pairs_neighbours():
    x = torch.zeros(3, 1, 6, dtype=F64)
    x[:, 0] = torch.tensor([1.0, 0.0, 0.0, 1.0, 5.0, 6.0], dtype=F64)
    y = P.rotate(x, {"base": 4.0, "dims": 4})
    a, b = 2.0, 2.0 * 0.5
    assert torch.allclose(y[2, 0], torch.tensor([math.cos(a), math.sin(a), -math.sin(b), math.cos(b), 5.0, 6.0], dtype=F64))
    assert torch.equal(y[0], x[0])


# --------------------------------------------------------------------------- the plain functions, by hand
def test_plain_dyn_tanh():
    w = {"n": torch.tensor([2.0, -1.0], dtype=F64), "n.b": torch.tensor([0.5, 0.25], dtype=F64), "n.alpha": torch.tensor(0.5, dtype=F64)}
    y = P.dyn_tanh(torch.tensor([[2.0, -4.0]], dtype=F64), w, "n")
    assert y[0].tolist() == pytest.approx([2.0 * math.tanh(1.0) + 0.5, math.tanh(2.0) + 0.25])


def test_plain_pair_rows():
    assert P.bigram_rows([5, 7, 5, 0], 10, 3, 4) == [10, (15 + 28) % 10, (21 + 20) % 10, 15 % 10]
    assert P.bigram_rows([9], 1, 3, 4) == [1]


def test_plain_sink_counts_once_and_is_not_scaled():
    s = torch.tensor([[0.0, -5.0], [math.log(2.0), math.log(3.0)]], dtype=F64)
    w = P.softmax_with_sink(s, P.causal(2), torch.tensor(math.log(5.0), dtype=F64))
    assert w[0].tolist() == pytest.approx([1.0 / 6.0, 0.0]) and w[1].tolist() == pytest.approx([0.2, 0.3])
    assert P.softmax_with_sink(s, P.causal(2))[1].tolist() == pytest.approx([0.4, 0.6])


def test_plain_choice_by_hand():
    """Groups of two; a group is worth both of its scores together, and what is left out counts as minus infinity."""
    s = torch.tensor([0.9, 0.1, 0.6, 0.6, 0.5, 0.2], dtype=F64)
    zero = torch.zeros(6, dtype=F64)
    assert P.choose(s, zero, 2, {"count": 3, "keep": 1}) == ([2, 3], pytest.approx(0.2))          # (worth 1.2 against 1.0)
    assert P.choose(s, zero, 3, {"count": 3, "keep": 2})[0] == [0, 2, 3]
    assert P.choose(s, zero, 2, None)[0] == [0, 2]
    low = torch.tensor([-2.0, -2.0, -2.0, -2.0, -1.0, -1.0], dtype=F64)
    assert P.choose(s, low, 2, {"count": 3, "keep": 1})[0] == [4, 5]         # choice scores below 0: no 0 of another group wins
    assert P.choose(s, low, 3, {"count": 3, "keep": 2})[0] == [4, 5, 2]
    assert P.choose(torch.tensor([0.3, 0.8, 0.5], dtype=F64), zero[:3], 2, {"count": 3, "keep": 2})[0] == [1, 2]      # groups of one


def test_plain_router_weights_are_plain_scores():
    x = torch.eye(2, dtype=F64)
    w = {"router": torch.tensor([[0.0, 1.0], [2.0, 0.0], [-1.0, 3.0]], dtype=F64), "correction": torch.tensor([0.0, 0.0, 5.0], dtype=F64)}
    idx, wt = P.route(x, w, "", {"top": 2})
    sg = lambda z: 1.0 / (1.0 + math.exp(-z))
    assert idx.tolist() == [[2, 1], [2, 0]]
    assert wt[0].tolist() == pytest.approx([sg(-1) / (sg(-1) + sg(2)), sg(2) / (sg(-1) + sg(2))])


def test_plain_layers_share_tensors_and_differ_in_state(tmp_path):
    folder = write_model(LELUTAR_A, str(tmp_path / "m"), 3)
    cfg, w = P.load(folder)
    assert [P.tensors_of(cfg, i) for i in range(7)] == [0, 1, 2, 2, 1, 2, 6]
    y = P.forward(cfg, w, [3, 5, 9])
    w2 = {k: (v * 2.0 if k == "l2.mix.o" else v) for k, v in w.items()}
    assert (P.forward(cfg, w2, [3, 5, 9]) - y).abs().max() > 1e-2
    w3 = dict(w, bigram=w["bigram"] * 0.0)
    d = (P.forward(cfg, w3, [3, 5, 9]) - y).abs().max(dim=1).values
    assert d.min() > 1e-3          # (the first token reads the table too: its last row)


def test_command_line_writes_and_lists_a_random_model(tmp_path, capsys):
    from ferrum_b200 import cli
    cfg = tmp_path / "cfg.json"
    cfg.write_text(json.dumps(LELUTAR_B))
    out = tmp_path / "model"
    assert cli.main(["random-weights", "--config", str(cfg), "--out", str(out), "--seed", "3", "--dtype", "bfloat16"]) == 0
    capsys.readouterr()
    assert cli.main(["dump", str(out)]) == 0
    listing = capsys.readouterr().out
    assert "l2.mix.uk [48, 96] bfloat16" in listing and "l1.mix.sink [20] float32" in listing and "l0." not in listing
    c, w = P.load(str(out))
    assert c["architecture"] == "Lelutar" and w["bigram"].shape == (101, 128)
