"""Tikunex without a GPU: configuration, tensor names, cache layout, kept pages, and hand-worked anchors of the plain
implementation's functions."""
import copy
import math

import pytest
import torch

import plain_tikunex as P
from tikunex_configs import TIKUNEX_A, TIKUNEX_B, TIKUNEX_C, TIKUNEX_D, write_model

from ferrum_b200 import host
from ferrum_b200.config import registry
from ferrum_b200.config.tikunex import GlaSpec, PairSpec, TikunexConfig
from ferrum_b200.errors import ConfigError, WeightsError

F64 = torch.float64


def test_config_reads_every_size_and_constant():
    c = TikunexConfig.from_dict(TIKUNEX_A)
    assert (c.n_vocab, c.n_embd, c.norm_eps, c.n_layer, c.side_dim) == (197, 52, 1e-5, 4, 6)
    assert (c.loop.start, c.loop.stop, c.loop.times) == (1, 3, 3)
    assert c.run_order() == [(0, False)] + [(1, True), (2, False)] * 3 + [(3, False)]
    pair, gla = c.layers[0].mixer, c.layers[1].mixer
    assert isinstance(pair, PairSpec) and isinstance(gla, GlaSpec)
    a, r = pair.left, pair.right
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.window, a.keep_first) == (3, 1, 10, 14, 0.4, 19, 3)
    assert (r.heads, r.dim, r.decay_rank, pair.left_scale, pair.right_scale) == (5, 6, 3, 0.7, 1.6)
    assert (gla.heads, gla.dim, gla.vdim, gla.tau, gla.decay_rank) == (3, 10, 14, 4.0, 5)
    assert c.layers[1].mlp is None and (c.layers[0].mlp.ff, c.layers[0].mlp.experts, c.layers[0].mlp.top) == (20, 5, 3)
    cc = TikunexConfig.from_dict(TIKUNEX_C)
    assert cc.loop is None and cc.side_dim == 0 and cc.run_order() == [(0, False), (1, False)]
    d = TikunexConfig.from_dict(TIKUNEX_D)
    assert d.layers[1].mixer.left.window == 0 and d.layers[0].mixer.left.keep_first == 0 and d.layers[1].mixer.right_scale == -0.9
    assert d.run_order() == [(0, False), (1, False), (2, True)]
    e = copy.deepcopy(TIKUNEX_B)
    e["layers"][0]["mixer"].pop("decay_rank")
    assert TikunexConfig.from_dict(e).layers[0].mixer.decay_rank is None          # the tensors' shapes decide then


@pytest.mark.parametrize("edit,message", [
    (lambda d: d["layers"][0].update(type="mamba2"), "not a mixer"),
    (lambda d: d["layers"][0]["mixer"]["left"]["mask"].update(size=0), "mask"),
    (lambda d: d["layers"][0]["mixer"]["left"].update(kv_heads=2), "kv_heads"),
    (lambda d: d["layers"][0]["mixer"].pop("right"), "right"),
    (lambda d: d["layers"][0]["mixer"].pop("left_scale"), "left_scale"),
    (lambda d: d["layers"][1]["mixer"].pop("tau"), "tau"),
    (lambda d: d["layers"][1]["mixer"].update(tau=0.0), "tau"),
    (lambda d: d["layers"][2]["mlp"]["router"].update(top=6), "experts"),
    (lambda d: d["layers"][2]["mlp"].update(kind="dense"), "feed-forward"),
    (lambda d: d["loop"].update(stop=5), "loop"),
    (lambda d: d["loop"].update(times=0), "loop"),
    (lambda d: d.pop("width"), "width"),
    (lambda d: d["token_side"].pop("dim"), "token_side"),
])
def test_config_refusals(edit, message):
    d = copy.deepcopy(TIKUNEX_A)
    edit(d)
    with pytest.raises(ConfigError, match=message):
        TikunexConfig.from_dict(d)


def build(d, dtype=torch.float32):
    arch = registry.lookup("Tikunex")
    return arch.build(arch.read_config(d), dtype, "cpu"), arch


@pytest.mark.parametrize("d", [TIKUNEX_A, TIKUNEX_B, TIKUNEX_C, TIKUNEX_D])
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
    assert ("loop.in" in w) == ("loop" in d) and ("side.embed" in w) == ("token_side" in d)
    for i, layer in enumerate(d["layers"]):
        assert (f"l{i}.norm2" in w) == (f"l{i}.mlp.router" in w) == (layer["mlp"] is not None)
    load_weights(model, folder, names, device="cpu")
    path = folder + "/model.safetensors"
    st = SafetensorsFile(path)
    tensors = {n: st.tensor(n).clone() for n in st.names()}
    tensors["l9.mix.q"] = tensors.pop("embed.norm")
    tensors["head"] = tensors["head"][:, :-1].contiguous()
    write_safetensors(path, tensors, {"format": "pt"})
    with pytest.raises(WeightsError) as err:
        load_weights(build(d)[0], folder, names, device="cpu")
    assert all(s in str(err.value) for s in ("missing: embed.norm", "unexpected: l9.mix.q", "head: shape"))


def test_inner_sizes_come_from_the_tensors(tmp_path):
    """Without `decay_rank` the file decides; two matrices that disagree are refused."""
    from ferrum_b200.weights import load_weights
    from ferrum_b200.weights.safetensors_io import SafetensorsFile, write_safetensors
    folder = write_model(TIKUNEX_A, str(tmp_path / "m"), 3)
    d = copy.deepcopy(TIKUNEX_A)
    for layer in d["layers"]:
        m = layer["mixer"]
        m.pop("decay_rank", None)
        m.get("right", {}).pop("decay_rank", None)
    model, arch = build(d)
    load_weights(model, folder, arch.hf_names(arch.read_config(d)), device="cpu")
    assert model.blocks[1].mixer.rank == 5 and model.blocks[0].mixer.right.rank == 3
    path = folder + "/model.safetensors"
    st = SafetensorsFile(path)
    tensors = {n: st.tensor(n).clone() for n in st.names()}
    tensors["l0.mix.right.w2"] = tensors["l0.mix.right.w2"][:, :2].contiguous()
    write_safetensors(path, tensors, {"format": "pt"})
    with pytest.raises(ValueError, match="inner size"):
        load_weights(build(d)[0], folder, arch.hf_names(arch.read_config(d)), device="cpu")


def test_every_pass_of_the_loop_has_planes_and_states_of_its_own():
    from ferrum_b200.cache.storage import CacheLayout
    model, _ = build(TIKUNEX_A)
    lay = CacheLayout(model)
    assert [r.block for r in model.schedule] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [r.before for r in model.schedule] == [None, 0, None, 0, None, 0, None, None]
    assert lay.group_keys == [(1, 14, 19, 2)] and lay.group_keep_first == [3]      # (kv heads, max(dim, vdim), window, parts)
    assert lay.run_plane == [0, None, 1, None, 2, None, 3, None] and lay.run_state == list(range(8))
    sizes = {0: 5 * 6 * 6 + 52, 1: 3 * 10 * 14, 2: 5 * 6 * 6 + 52, 3: 3 * 10 * 14}  # S, and the last token's row of the recurrence behind shifts
    assert [n.shape[0] for n in lay.state_needs] == [sizes[r.block] for r in model.schedule]
    lay = CacheLayout(build(TIKUNEX_D)[0])
    assert lay.group_keys == [(4, 20, 7, 2), (1, 16, 0, 2)] and lay.group_keep_first == [0, 0]


def test_groups_differ_by_the_kept_first_keys():
    from ferrum_b200.cache.storage import CacheLayout
    d = copy.deepcopy(TIKUNEX_A)
    d["layers"][2] = copy.deepcopy(d["layers"][2])
    d["layers"][2]["mixer"]["left"]["mask"]["keep_first"] = 11
    lay = CacheLayout(build(d)[0])
    assert lay.group_keys == [(1, 14, 19, 2)] * 2 and lay.group_keep_first == [3, 11]
    assert lay.run_group[0] == 0 and lay.run_group[2] == 1


@pytest.mark.parametrize("keep,page,window", [(3, 8, 20), (8, 8, 20), (9, 8, 20), (17, 4, 6), (1, 16, 1), (40, 8, 20)])
def test_kept_pages_stay_and_the_others_leave(keep, page, window):
    h = host.module()
    pages = 40
    m = h.CacheManager([h.GroupSpec(page, window, pages, 64, keep)], 2)
    s = m.open()
    n, kept = 0, -(-keep // page)
    for step in [1, 5, 1, 1, 30, 1, 1, 7, 40, 1, 1]:
        m.grow(s, n + step)
        m.commit(s, n + step)
        n += step
        first = max(0, n - window + 1) // page
        last = (n - 1) // page
        t = m.table(0, s)
        for lp in range(last + 1):
            assert (t[lp] >= 0) == (lp < kept or lp >= first), (n, lp)
        assert all(p < 0 for p in t[last + 1:]) and m.check() == ""
    assert m.pages_held(0, s) <= kept + (window - 1) // page + 2
    other = m.open()
    m.grow(other, page)
    m.commit(other, page)
    assert not set(p for p in m.table(0, s) if p >= 0) & set(p for p in m.table(0, other) if p >= 0)
    m.close(s)
    m.close(other)
    assert m.free_pages(0) == pages and m.check() == ""


# --------------------------------------------------------------------------- the plain functions, by hand
def test_plain_mask():
    m = P.sink_window_mask(9, 3, 2)
    assert [j for j in range(9) if m[8, j]] == [0, 1, 6, 7, 8] and [j for j in range(9) if m[3, j]] == [0, 1, 2, 3]
    assert [j for j in range(9) if m[1, j]] == [0, 1] and [j for j in range(9) if m[4, j]] == [0, 1, 2, 3, 4]
    assert torch.equal(P.sink_window_mask(5, 0, 0), torch.tril(torch.ones(5, 5, dtype=torch.bool)))
    assert [j for j in range(5) if P.sink_window_mask(5, 1, 0)[4, j]] == [4]


def test_plain_norm_and_blend():
    x = torch.tensor([[3.0, -4.0]], dtype=F64)
    r = 1.0 / math.sqrt(12.5)
    assert torch.allclose(P.centred_norm(x, torch.tensor([0.0, 1.0], dtype=F64), 0.0), torch.tensor([[3 * r, -8 * r]], dtype=F64))
    h = torch.tensor([[1.0, 2.0], [5.0, 10.0]], dtype=F64)
    mu = torch.tensor([0.25, 1.0], dtype=F64)
    assert torch.allclose(P.shifted_mix(h, mu), torch.tensor([[0.75, 0.0], [4.0, 2.0]], dtype=F64))


def test_plain_two_tokens_of_each_recurrence():
    """One head, keys of 2, one value column.  Gated linear attention reads after the write; the other form reads the old
    state plus the bonus times the current token, and decays before it writes."""
    k = torch.tensor([[1.0, 2.0], [3.0, 1.0]], dtype=F64)[:, None]
    q = torch.tensor([[1.0, 1.0], [2.0, -1.0]], dtype=F64)[:, None]
    v = torch.tensor([[10.0], [1.0]], dtype=F64)[:, None]
    a = torch.tensor([[0.9, 0.9], [0.5, 0.1]], dtype=F64)[:, None]
    # S1 = [10, 20]; S2 = [5 + 3, 2 + 1]
    assert P.gla_walk(q, k, v, a).flatten().tolist() == pytest.approx([30.0, 2 * 8 - 3])
    u = torch.tensor([[2.0, 0.5]], dtype=F64)
    # o1 = (2 * 1 + 0.5 * 2) * 10; S1 = [10, 20]; o2 = 2 (10 + 2 * 3) - (20 + 0.5 * 1)
    assert P.rwkv_walk(q, k, v, a, u).flatten().tolist() == pytest.approx([30.0, 32.0 - 20.5])


def test_plain_router_weighs_the_chosen_logits_only():
    x = torch.eye(3, dtype=F64)
    w = {"router": torch.tensor([[1.0, 0.0, 0.0], [0.0, 2.0, 0.0], [0.0, 0.0, 3.0], [0.5, 0.5, 0.5]], dtype=F64),
         "router.b": torch.tensor([0.0, 0.0, 0.0, 0.25], dtype=F64)}
    margins = []
    idx, wt = P.route(x, w, "", {"top": 2}, None, margins)
    assert idx.tolist() == [[0, 3], [1, 3], [2, 3]]
    assert wt[1].tolist() == pytest.approx([math.exp(2.0) / (math.exp(2.0) + math.exp(0.75)), math.exp(0.75) / (math.exp(2.0) + math.exp(0.75))])
    z = torch.tensor([1.0, 0.0, 0.0, 0.75], dtype=F64)
    assert float(margins[0][0]) == pytest.approx(0.75 / float(z.std()))


def test_plain_run_order():
    assert P.run_order(TIKUNEX_A) == TikunexConfig.from_dict(TIKUNEX_A).run_order()
    assert P.run_order(TIKUNEX_C) == [(0, False), (1, False)] and P.run_order(TIKUNEX_B) == [(0, True), (1, False)] * 2 + [(2, False)]
