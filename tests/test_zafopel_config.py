"""CPU tests of the Zafopel family: configuration, weight layout, cache geometry, what a prefill sees, page release, and the oracle itself."""
import copy
import math

import pytest
import torch

import dulisun_cases as D
import zafopel_cases as C
import zafopel_oracle as O
from rpeg_b200.engine.generation import PAGE, Generator, page_elems
from rpeg_b200.models.registry import config_from_hf, hf_config_dict, load_model, model_class
from rpeg_b200.models.served import ServedDecoder
from rpeg_b200.models.zafopel import DenseFF, InputScaledMixture, ZafopelModel, _Spans
from rpeg_b200.runtime.errors import RuntimeConfigError


def test_config_reads_every_size_and_round_trips():
    raw = C.unlike()
    cfg = config_from_hf(raw)
    assert model_class(cfg) is ZafopelModel and issubclass(ZafopelModel, ServedDecoder)
    assert (cfg.width, cfg.vocab, cfg.norm_eps, cfg.n_layers) == (100, 301, 1e-5, 5)
    a, b, c, d = (l.mixer for l in cfg.layers[:4])
    assert (a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.q_rank, a.scale, a.rot_base) == (5, 20, 12, 28, 36, 44, 0.3, 5000.0)
    assert a.sink and a.window == 0 and a.kv_from is None and not b.sink and b.window == 37 and b.q_rank == 0
    assert (c.kv_from, c.window, d.kv_from, d.window, d.sink) == (1, 100, 0, 0, True)
    assert cfg.layers[0].mlp == InputScaledMixture(6, 3, 36) and cfg.layers[1].mlp == DenseFF(50) and cfg.layers[3].mlp is None
    for name in ("unlike", "sliding", "wide"):
        raw = getattr(C, name)()
        assert hf_config_dict(config_from_hf(raw)) == raw and config_from_hf(hf_config_dict(config_from_hf(raw))) == config_from_hf(raw)
    # one padded latent row per token; nothing for a layer that reads another's
    assert cfg.kv_geometry() == [(1, 40 + 16, 0), (1, 48 + 8, 0), (0, 0, 0), (0, 0, 0), (1, 136 + 8, 0)]


@pytest.mark.parametrize("path,value,word", [
    (("layers", 0, "type"), "attention", "mixer type"), (("layers", 0, "mixer", "heads"), 0, "heads"), (("layers", 0, "mixer", "rot", "dims"), 10, "rot.dims"),
    (("layers", 1, "mixer", "rot_dim"), 7, "rot"), (("layers", 1, "mixer", "kv_rank"), 2000, "kv_rank"), (("layers", 1, "mixer", "mask", "size"), 0, "mask.size"),
    (("layers", 0, "mixer", "mask"), {"size": 4}, "causal"), (("layers", 0, "mixer", "q_rank"), 0, "q_rank"), (("layers", 2, "mixer", "kv_from"), 2, "kv_from"),
    (("layers", 2, "mixer", "kv_from"), 0, "kv_rank"), (("layers", 3, "mixer", "kv_from"), 2, "kv_from"), (("layers", 0, "mlp", "kind"), "other", "kind"),
    (("layers", 0, "mlp", "router", "top"), 7, "choose"), (("layers", 1, "mlp", "ff"), 0, "ff"), (("layers",), [], "no layers")])
def test_config_rejects_what_is_not_implemented(path, value, word):
    raw = copy.deepcopy(C.unlike())
    at = raw
    for p in path[:-1]:
        at = at[p]
    at[path[-1]] = value
    with pytest.raises(RuntimeConfigError, match=word):
        config_from_hf(raw)


def test_planner_and_training_refuse_the_family_with_a_reason():
    from rpeg_b200.runtime.hf import model_spec_from_hf_config
    with pytest.raises(RuntimeConfigError, match="cost model"):
        model_spec_from_hf_config(C.sliding())
    with pytest.raises(ValueError, match="no backward"):
        ZafopelModel(config_from_hf(C.sliding()), "cpu", trainable=True)


def test_weights_land_in_padded_layout(tmp_path):
    raw = C.unlike()
    t = C.tensors(raw, 3)
    m = load_model(D.write(raw, t, tmp_path / "m"), "cpu")
    p, w = m.p, 100
    # layer 0: query latent (44 -> 48 rows), latent (36 -> 40) and rotated part (12 -> 16), router (6 -> 8)
    w_in = p["l0.w_in"]
    assert w_in.shape == (48 + 40 + 16 + 8, 104)
    assert torch.equal(w_in[:44, :w], t["l0.mix.dq"]) and torch.equal(w_in[48:84, :w], t["l0.mix.dkv"][:36])
    assert torch.equal(w_in[88:100, :w], t["l0.mix.dkv"][36:]) and torch.equal(w_in[104:110, :w], t["l0.mlp.router"])
    assert w_in[44:48].abs().sum() == 0 and w_in[84:88].abs().sum() == 0 and w_in[100:104].abs().sum() == 0 and w_in[:, w:].abs().sum() == 0
    uq = p["l0.w_uq"].view(5, 24 + 16, 48)
    src = t["l0.mix.uq"].view(5, 32, 44)
    assert torch.equal(uq[:, :20, :44], src[:, :20]) and torch.equal(uq[:, 24:36, :44], src[:, 20:]) and uq[:, 20:24].abs().sum() == 0
    k, v = m._kv_maps(0)
    assert k.shape == (5, 24, 40) and v.shape == (5, 32, 40)
    assert torch.equal(k[:, :20, :36].reshape(100, 36), t["l0.mix.uk"]) and torch.equal(v[:, :28, :36].reshape(140, 36), t["l0.mix.uv"])
    assert torch.equal(p["l0.wo"].view(104, 5, 32)[:w, :, :28].reshape(w, 140), t["l0.mix.o"])
    # layers 2 and 3 have no latent of their own
    assert p["l2.w_in"].shape == (7 * 48 + 8, 104) and "l2.kv_norm" not in p and p["l3.w_in"].shape == (24, 104)
    gu = p["l0.w_gate_up"]
    assert gu.shape == (6, 80, 104) and torch.equal(gu[4, :36, :w], t["l0.mlp.e4.gate"]) and torch.equal(gu[4, 40:76, :w], t["l0.mlp.e4.up"])
    assert torch.equal(p["l0.w_down"][4, :w, :36], t["l0.mlp.e4.down"]) and torch.equal(m._ff_rows(1)[:50, :w], t["l1.mlp.up"])
    assert torch.equal(m.alpha.bfloat16(), torch.stack([t[f"l{i}.norm1.alpha"] for i in range(5)] + [t["final.norm.alpha"]]))
    assert torch.equal(p["l2.norm1.b"][:w], t["l2.norm1.b"]) and torch.equal(m.sink[3], t["l3.mix.sink"].float()) and m.sink[1] is None
    assert torch.equal(p["head"][:301, :w], t["head"]) and torch.equal(p["embed"][:301, :w], t["embed"])
    f32 = load_model(tmp_path / "m", "cpu", dtype=torch.float32)
    assert f32.w.dtype == torch.float32 and torch.equal(f32.w, m.w.float())
    assert m.lasting_caches() == {0, 1}


def test_loading_reports_missing_misshaped_and_unknown_tensors(tmp_path):
    raw = C.unlike()
    t = C.tensors(raw)
    for k, name in enumerate(("l0.mix.sink", "l1.norm1.alpha", "l4.mix.dkv.norm", "final.norm.b", "head")):
        with pytest.raises(RuntimeConfigError, match=f"{name} is missing"):
            load_model(D.write(raw, {n: v for n, v in t.items() if n != name}, tmp_path / f"a{k}"), "cpu")
    with pytest.raises(RuntimeConfigError, match="shape mismatch of l0.mix.uk"):
        load_model(D.write(raw, {**t, "l0.mix.uk": t["l0.mix.uv"].clone()}, tmp_path / "b"), "cpu")
    with pytest.warns(UserWarning, match="l2.mix.dkv"):       # a layer that reads another's latents has no place for its own
        load_model(D.write(raw, {**t, "l2.mix.dkv": torch.ones(3)}, tmp_path / "c"), "cpu")


def test_first_visible_key_follows_the_longest_window():
    m = ZafopelModel(config_from_hf(C.sliding()), "cpu", seed=None)
    assert [m.first_visible_key(p) for p in (0, 89, 90, 91, 300)] == [0, 0, 1, 2, 211]
    assert ZafopelModel(config_from_hf(C.unlike()), "cpu", seed=None).first_visible_key(500) == 0     # a causal layer reads everything


@pytest.mark.parametrize("window", [0, 1, 2, 7, 64, 1000])
def test_spans_count_rows_and_pairs(window):
    starts, lens = [0, 5, 63, 200, 3], [9, 2, 130, 1, 1]
    s = _Spans(starts, lens, "cpu")
    mask = O.visible(400, window or None)
    total, off, lo = s.rows(window)
    want_lo, want_off, pairs = [], [0], 0
    for a, n in zip(starts, lens):
        seen = mask[a:a + n].nonzero()[:, 1]
        want_lo.append(int(seen.min()))
        want_off.append(want_off[-1] + a + n - int(seen.min()))
        pairs += int(mask[a:a + n].sum())
    assert total == s.total(window) == want_off[-1] and off.tolist() == want_off and lo.tolist() == want_lo and s.pairs(window) == pairs


def test_generator_carves_a_cache_without_values():
    """Layers without a cache of their own and without values take no bytes; pages cover every layer that has one."""
    cfg = config_from_hf(C.unlike())
    model = type("M", (), dict(cfg=cfg, device=torch.device("cpu"), dtype=torch.float32, cached_prefill=True))()
    gen = Generator(model, max_slots=2, max_seq_len=128, kv_budget_bytes=5 * page_elems(cfg.kv_geometry()) * 4, use_graphs=False)
    assert page_elems(cfg.kv_geometry()) == PAGE * (56 + 56 + 144) and gen.pool.num_pages == 5
    assert [tuple(c.shape) for c in gen.kcache] == [(5, 1, PAGE, 56), (5, 1, PAGE, 56), (5, 0, PAGE, 0), (5, 0, PAGE, 0), (5, 1, PAGE, 144)]
    assert all(v.numel() == 0 for v in gen.vcache) and gen.kv_storage.numel() == 5 * PAGE * 256


def test_scratch_caches_of_whole_sequences_keep_what_later_layers_read():
    m = ZafopelModel(config_from_hf(C.unlike()), "cpu", seed=None)
    kc, _ = m._scratch_cache(3)
    kc[0].fill_(1.0)
    kc[1].fill_(2.0)
    kc[4].fill_(3.0)
    assert (kc[0] == 1).all() and (kc[1] == 2).all()


def test_oracle_mechanisms():
    """The oracle against hand-checkable cases."""
    F = torch.float64
    assert [sorted(r.nonzero()[:, 0].tolist()) for r in O.visible(5, 2)] == [[0], [0, 1], [1, 2], [2, 3], [3, 4]]
    assert O.visible(3, None).tolist() == [[True, False, False], [True, True, False], [True, True, True]]
    x = torch.randn(4, 2, 6, dtype=F)
    r = O.rotate(x, torch.arange(4), 100.0)
    assert torch.equal(r[0], x[0]) and torch.allclose(r.pow(2).sum(-1), x.pow(2).sum(-1))
    a = 3 * 100.0 ** (-2.0 / 6)
    assert torch.allclose(r[3, 0, 2], x[3, 0, 2] * math.cos(a) - x[3, 0, 3] * math.sin(a))
    t = {"n": torch.tensor([2.0, 2.0], dtype=F), "n.b": torch.tensor([0.5, 0.5], dtype=F), "n.alpha": torch.tensor(3.0, dtype=F)}
    assert torch.allclose(O.dynamic_tanh(torch.tensor([[0.0, 100.0]], dtype=F), t, "n"), torch.tensor([[0.5, 2.5]], dtype=F))
    # a sink as large as the only key's score halves the output
    q = torch.ones(1, 1, 4, dtype=F)
    assert torch.allclose(O.attend(q, q, q, torch.ones(1, 1, dtype=torch.bool), 0.5, torch.tensor([2.0], dtype=F)), 0.5 * q)
    # scores weigh the inputs: with a linear region's worth of input the squared gate shows it (silu(w g) w u, not w silu(g) u)
    m = {"router": {"experts": 2, "top": 1}}
    t = {"router": torch.tensor([[1.0], [-1.0]], dtype=F), "e0.gate": torch.tensor([[1.0]], dtype=F), "e0.up": torch.tensor([[1.0]], dtype=F),
         "e0.down": torch.tensor([[1.0]], dtype=F), "e1.gate": torch.zeros(1, 1, dtype=F), "e1.up": torch.zeros(1, 1, dtype=F), "e1.down": torch.zeros(1, 1, dtype=F)}
    sg = lambda z: 1 / (1 + math.exp(-z))  # noqa: E731
    z = sg(2.0) * 2.0
    assert torch.allclose(O.moe(torch.tensor([[2.0]], dtype=F), t, "", m), torch.tensor([[z * sg(z) * z]], dtype=F))
    assert torch.allclose(O.dense(torch.tensor([[-3.0], [3.0]], dtype=F), {"up": torch.ones(1, 1, dtype=F), "down": torch.ones(1, 1, dtype=F)}, ""),
                          torch.tensor([[0.0], [9.0]], dtype=F))
