"""CPU tests of the Dulisun family: configuration, weight layout, and the page and position accounting of sessions."""
import copy
import json

import pytest
import torch

import dulisun_cases as C
import dulisun_oracle as O
from rpeg_b200.engine.generation import PAGE, Generator, page_elems
from rpeg_b200.engine.session import Session
from rpeg_b200.models.dulisun import DulisunModel
from rpeg_b200.models.registry import config_from_hf, hf_config_dict, load_model, model_class
from rpeg_b200.ops import kernels as K
from rpeg_b200.runtime.errors import RuntimeConfigError


def test_config_reads_every_size_and_round_trips():
    raw = C.unlike()
    cfg = config_from_hf(raw)
    assert model_class(cfg) is DulisunModel and (cfg.width, cfg.vocab, cfg.norm_eps, cfg.n_layers) == (100, 301, 1e-5, 4)
    m, e = cfg.layers[0].mixer, cfg.layers[0].mlp
    assert (m.heads, m.kv_heads, m.dim, m.window, m.rot_dims, m.rot_base, m.scale) == (6, 3, 20, 50, 12, 5000.0, 0.3)
    assert (e.experts, e.top, e.ff, e.shared_ff, e.groups, e.keep, e.n_shared) == (6, 3, 36, 50, 3, 2, 2)
    assert cfg.layers[1].mlp is None and cfg.layers[2].mixer.window == 0 and cfg.layers[2].mixer.rot_dims == 0
    assert cfg.layers[2].mlp.n_shared == 0 and cfg.layers[2].mlp.groups == 1
    assert config_from_hf(hf_config_dict(cfg)) == cfg
    assert cfg.kv_geometry() == [(3, 24, 24), (1, 40, 40), (4, 136, 136), (2, 64, 64)]


def test_planner_refuses_the_family_with_a_reason():
    from rpeg_b200.runtime.hf import model_spec_from_hf_config
    with pytest.raises(RuntimeConfigError, match="cost model"):
        model_spec_from_hf_config(C.regular())


@pytest.mark.parametrize("path,value,word", [
    (("layers", 0, "type"), "recurrent", "mixer type"), (("layers", 0, "mixer", "kv_heads"), 4, "divide"),
    (("layers", 0, "mixer", "vdim"), 24, "vdim"), (("layers", 0, "mixer", "dim"), 300, "dim"), (("layers", 0, "mixer", "rot", "dims"), 13, "rot"),
    (("layers", 0, "mlp", "kind"), "dense", "kind"), (("layers", 0, "mlp", "router", "experts"), 7, "groups"),
    (("layers", 0, "mlp", "router", "top"), 5, "choose"), (("architecture",), "Other", "architecture"), (("layers",), [], "no layers")])
def test_config_rejects_what_is_not_implemented(path, value, word):
    raw = copy.deepcopy(C.unlike())
    at = raw
    for p in path[:-1]:
        at = at[p]
    at[path[-1]] = value
    with pytest.raises(RuntimeConfigError, match=word):
        config_from_hf(raw)


def test_weights_land_in_padded_layout(tmp_path):
    raw = C.unlike()
    t = C.tensors(raw, 3)
    m = load_model(C.write(raw, t, tmp_path / "m"), "cpu")
    cfg = m.cfg
    q = m.p["l0.wqk"].view(9, 24, 104)                       # 6 query heads, then 3 key heads
    assert torch.equal(q[:6, :20, :100].reshape(120, 100), t["l0.mix.q"]) and torch.equal(q[6:, :20, :100].reshape(60, 100), t["l0.mix.k"])
    assert q[:, 20:].abs().sum() == 0 and q[..., 100:].abs().sum() == 0
    assert torch.equal(m.p["l0.wo"].view(104, 6, 24)[:100, :, :20].reshape(100, 120), t["l0.mix.o"])
    up, down = m.p["l0.w_up"], m.p["l0.w_down"]
    assert up.shape == (8, 40, 104) and down.shape == (8, 104, 40)
    assert torch.equal(up[4, :36, :100], t["l0.mlp.e4.up"]) and torch.equal(down[4, :100, :36], t["l0.mlp.e4.down"])
    # the shared part of 50 hidden units fills two always-on experts of 36
    assert torch.equal(torch.cat([up[6, :36, :100], up[7, :14, :100]]), t["l0.mlp.shared.up"]) and up[7, 14:].abs().sum() == 0
    assert torch.equal(torch.cat([down[6, :100, :36], down[7, :100, :14]], 1), t["l0.mlp.shared.down"])
    assert torch.equal(m.sink[3], t["l3.mix.sink"].float()) and torch.equal(m.p["embed"][:301, :100], t["embed"])
    f32 = load_model(tmp_path / "m", "cpu", dtype=torch.float32)
    assert f32.w.dtype == torch.float32 and torch.equal(f32.w, m.w.float())
    assert m.first_visible_key(129) == 0 and cfg.layers[2].mixer.window == 0


def test_loading_reports_missing_misshaped_and_unknown_tensors(tmp_path):
    raw = C.regular()
    t = C.tensors(raw)
    with pytest.raises(RuntimeConfigError, match="l1.mix.sink is missing"):
        load_model(C.write(raw, {n: v for n, v in t.items() if n != "l1.mix.sink"}, tmp_path / "a"), "cpu")
    with pytest.raises(RuntimeConfigError, match="shape mismatch of l0.mix.k"):
        load_model(C.write(raw, {**t, "l0.mix.k": t["l0.mix.q"].clone()}, tmp_path / "b"), "cpu")
    with pytest.warns(UserWarning, match="l9.extra"):
        load_model(C.write(raw, {**t, "l9.extra": torch.ones(3)}, tmp_path / "c"), "cpu")
    with pytest.raises(ValueError, match="no backward"):
        DulisunModel(config_from_hf(raw), "cpu", trainable=True)


def test_oracle_mechanisms():
    """The oracle against hand-checkable cases."""
    m = O.visible(7, 3)
    assert [sorted(m[i].nonzero()[:, 0].tolist()) for i in (0, 2, 3, 5, 6)] == [[0], [0, 1, 2], [3], [3, 4, 5], [6]]
    x = torch.randn(5, 1, 6, dtype=torch.float64)
    r = O.rotate(x, torch.arange(5), 100.0, 4)
    assert torch.equal(r[0], x[0]) and torch.equal(r[..., 4:], x[..., 4:]) and not torch.allclose(r[1, 0, :4], x[1, 0, :4])
    assert torch.allclose(r.pow(2).sum(-1), x.pow(2).sum(-1))
    # a sink as large as the only key's score halves the output
    q = torch.ones(1, 1, 4, dtype=torch.float64)
    out = O.attend(q, q, q, torch.ones(1, 1, dtype=torch.bool), 0.5, torch.tensor([2.0], dtype=torch.float64))
    assert torch.allclose(out, 0.5 * q)
    # expert 5 has the largest score, so group 1 wins although group 0 holds the next three
    assert O.route([0.2, 0.19, 0.18, 0.0, 0.01, 0.4], {"experts": 6, "top": 2, "groups": {"count": 2, "keep": 1}}) == [5, 4]
    assert O.route([0.2, 0.19, 0.18, 0.0, 0.01, 0.4], {"experts": 6, "top": 2}) == [5, 0]


# --------------------------------------------------------------------------- sessions on a stand-in model
class _Cfg:
    vocab = 1000

    def __init__(self, windows):
        self.windows = windows

    def kv_geometry(self, tp=1):
        return [(1, 8, 8)] * len(self.windows)


class _Counter:
    """Stands in for a model: 'attention' adds up the token ids it finds in the cache inside the row's chunk, so a wrong
    position, page or chunk edge changes the result. Reading a page the row does not own finds somebody else's ids."""
    dtype = torch.float32
    device = torch.device("cpu")
    cached_prefill = True

    def __init__(self, windows):
        self.cfg = _Cfg(windows)

    def first_visible_key(self, pos):
        return min(pos // w * w if w else 0 for w in self.cfg.windows)

    def _rows(self, tokens, pos, slot, table, kcache):
        for t, p, s in zip(tokens.tolist(), pos.tolist(), slot.tolist()):
            for c in kcache:
                c[int(table[s, p // PAGE]), 0, p % PAGE, 0] = float(t)
        out = []
        for p, s in zip(pos.tolist(), slot.tolist()):
            total = 0.0
            for c, w in zip(kcache, self.cfg.windows):
                for j in range(p // w * w if w else 0, p + 1):
                    page = int(table[s, j // PAGE])
                    assert page > 0, "a visible key's page was given back"
                    total += float(c[page, 0, j % PAGE, 0])
            out.append(total)
        return torch.tensor(out)[:, None]

    def prefill(self, tokens, pos, cu, max_len, slot, table, kcache, vcache):
        assert max_len == int((cu[1:] - cu[:-1]).max())
        return self._rows(tokens, pos, slot, table, kcache)

    def decode_step(self, token, pos, slot_ids, seq_len, table, kcache, vcache, nsplit=1, groups=None):
        assert torch.equal(seq_len, pos + 1)
        return self._rows(token, pos, slot_ids, table, kcache)

    def lm_logits(self, xf, decode=False):
        return xf


def _expected(tokens, windows):
    return [float(sum(sum(tokens[(p // w * w if w else 0):p + 1]) for w in windows)) for p in range(len(tokens))]


@pytest.mark.parametrize("windows", [(100,), (64, 192), (50, 0), (10, 30)])
def test_session_positions_pages_and_reuse(windows, monkeypatch):
    monkeypatch.setattr(K, "gather_rows", lambda x, rows: x[rows.long()])
    model = _Counter(windows)
    gen = Generator(model, max_slots=4, max_seq_len=512, kv_budget_bytes=20 * page_elems(model.cfg.kv_geometry()) * 4, use_graphs=False)
    s = Session(gen)
    total = s.gen.pool.available()
    g = torch.Generator().manual_seed(1)
    for rnd in range(4):                                   # later rounds run on slots and pages that were used before
        seqs = {f"{rnd}.{i}": torch.randint(1, 1000, (n,), generator=g).tolist() for i, n in enumerate((301, 130, 65))}
        done = {k: 0 for k in seqs}
        got = {k: [] for k in seqs}
        while any(done[k] < len(v) for k, v in seqs.items()):
            step = []
            for k, v in seqs.items():
                left = len(v) - done[k]
                if left and torch.rand(1, generator=g).item() < 0.7:
                    n = min(left, int((1, 1, 2, 3, 17, 64, 90)[int(torch.randint(0, 7, (1,), generator=g))]))
                    step.append((k, v[done[k]:done[k] + n], list(range(n))))
                    done[k] += n
            if not step:
                continue
            for (k, _, _), out in zip(step, s.feed(step)):
                got[k] += out[:, 0].tolist()
        for k, v in seqs.items():
            assert got[k] == _expected(v, windows), k
        if all(windows):                                   # passed pages went back while the requests were still live
            for k, q in s.requests.items():
                assert q.gone == min(model.first_visible_key(len(seqs[k])) // PAGE, -(-len(seqs[k]) // PAGE))
        for k in seqs:
            s.end(k)
        assert gen.pool.available() == total and len(s.free_slots) == 4 and not s.requests


def test_session_refuses_bad_steps(monkeypatch):
    monkeypatch.setattr(K, "gather_rows", lambda x, rows: x[rows.long()])
    model = _Counter((64,))
    gen = Generator(model, max_slots=2, max_seq_len=128, kv_budget_bytes=1e6, use_graphs=False)
    s = Session(gen)
    for bad, word in (([("a", [], [])], "no tokens"), ([("a", [1000], [])], "vocabulary"), ([("a", [1], [1])], "place"),
                      ([("a", [1], []), ("a", [2], [])], "once"), ([("a", [1] * 129, [])], "max_seq_len")):
        with pytest.raises(ValueError, match=word):
            s.feed(bad)
    assert s.feed([("b", [7, 8], [])]) == [None]
    with pytest.raises(RuntimeError, match="slots"):
        s.feed([("c", [1], []), ("d", [1], [])])
    assert set(s.requests) == {"b"}                        # a refused step leaves nothing behind


def test_generator_refuses_portions_without_cached_prefill():
    model = _Counter((64,))
    model.cached_prefill = False
    with pytest.raises(ValueError, match="whole prompts"):
        Generator(model, max_slots=2, max_seq_len=128, kv_budget_bytes=1e6, prefill_portion=16)


def test_on_demand_build_compiles_named_sources_only(tmp_path, monkeypatch):
    """``ensure`` on a tree without built files compiles the family's sources and nothing else; with an up-to-date full
    library it compiles nothing."""
    from rpeg_b200 import build_ext as B
    built = []
    csrc = tmp_path / "csrc"
    csrc.mkdir()
    for n in ("a.cu", "b.cu", "c.cu"):
        (csrc / n).write_text("")
    for name, v in (("PKG", tmp_path), ("CSRC", csrc), ("LIB", tmp_path / "full.so"), ("PART_LIB", tmp_path / "part.so")):
        monkeypatch.setattr(B, name, v)

    def compile_(src, verbose):
        built.append(src.name)
        src.with_suffix(".o").write_text("")
        return src.with_suffix(".o"), ""

    monkeypatch.setattr(B, "_compile", compile_)
    monkeypatch.setattr(B.subprocess, "run", lambda cmd, **kw: (open(cmd[cmd.index("-o") + 1], "w").close(), type("R", (), {"returncode": 0})())[1])
    assert B.ensure(["a.cu", "c.cu"]) == tmp_path / "part.so" and sorted(built) == ["a.cu", "c.cu"]
    assert B.ensure(["a.cu", "c.cu"]) == tmp_path / "part.so" and len(built) == 2
    assert B.ensure(None) == tmp_path / "full.so" and sorted(built) == ["a.cu", "b.cu", "c.cu"]
    assert B.ensure(["a.cu"]) == tmp_path / "full.so" and len(built) == 3
    assert json.dumps(sorted(p.name for p in tmp_path.glob("*.so"))) == '["full.so", "part.so"]'
