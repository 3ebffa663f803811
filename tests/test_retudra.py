"""Retudra through the engine against the plain implementation (``plain_retudra``): every way of
cutting the same requests into steps, in 32-bit and bfloat16, on configurations that differ in every
size, in the order of their layers and in their constants."""
import copy
import io
import json
import math

import pytest
import torch

import plain_retudra as plain
import replay
from tiny_retudra import CONFIGS, RA, RC, make_folder
from tolerances import SPLITS, VS_PLAIN, rel_err

F64 = torch.float64


# ---------------------------------------------------------------- configuration (no GPU)

def test_config_round_trip_and_registry():
    from airframe_b200.config import RetudraConfig, config_from_dict
    cfg = config_from_dict(RA)
    assert isinstance(cfg, RetudraConfig)
    assert config_from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg
    spec = cfg.model_spec()
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 3, 4]
    assert [(layer.block.kind, layer.mixer.kind, layer.feed_forward.kind) for layer in spec.layers] == \
        [("postnorm", "channel_delta", "routed_experts"), ("postnorm", "attention", "gated_mlp"),
         ("postnorm", "latent_attention", "none"), ("postnorm", "attention", "routed_experts"),
         ("postnorm", "channel_delta", "gated_mlp")]
    assert spec.layers[1].norms["post_mixer"].params == {"weight": "l1.norm1", "bias": "l1.norm1.b", "size": 72, "eps": 1e-5,
                                                         "scale": 0.6}
    assert spec.layers[2].norms.keys() == {"post_mixer", "post_side"}
    assert spec.layers[3].norms["post_side"].params["scale"] == 0.6 and spec.layers[3].norms["post_side"].params["weight"] == "l3.side.norm"
    side = spec.layers[3].block.params["side"].params
    assert (side["dim"], side["index"], side["parts"], side["table_weight"]) == (12, 3, 5, "side.embed")
    delta = spec.layers[0].mixer.params
    assert (delta["num_heads"], delta["num_kv_heads"], delta["head_dim"], delta["value_dim"], delta["taps"]) == (4, 2, 12, 20, 3)
    assert delta["weights"]["k_conv"] == "l0.mix.k.conv" and delta["weights"]["A_log"] == "l0.mix.A_log"
    at = spec.layers[3].mixer.params
    assert (at["window"], at["keep_first"], at["qk_norm"]["whole"], at["scale"]) == (70, 67, True, 0.2)
    assert (at["position"].params["pairing"], at["position"].params["rotary_dim"], at["position"].params["theta"]) == ("half", 18, 900.0)
    lat = spec.layers[2].mixer.params
    assert (lat["num_heads"], lat["head_dim"], lat["rot_dim"], lat["value_dim"], lat["kv_rank"]) == (3, 10, 6, 14, 20)
    assert lat["window"] is None and lat["value_gate_weight"] == "l2.mix.g" and "q_rank" not in lat
    ro = spec.layers[0].feed_forward.params["router"]
    assert (ro["score"], ro["group_score"], ro["identity"], ro["groups"]) == ("softmax", "max", 2, {"count": 3, "keep": 2})
    assert spec.head.params["weight"] == "head" and spec.head.params["softcap"] == 9.0
    other = config_from_dict(RC).model_spec()
    assert other.head.params["softcap"] == 0.0 and "side" not in other.layers[0].block.params
    assert other.layers[1].mixer.params["window"] is None and other.layers[1].mixer.params["keep_first"] == 0


def test_config_refuses_what_it_does_not_know():
    from airframe_b200.config import ConfigError, config_from_dict

    def broken(edit):
        d = copy.deepcopy(RA)
        edit(d)
        with pytest.raises(ConfigError):
            config_from_dict(d)

    broken(lambda d: d["layers"][0].update(type="general_delta"))
    broken(lambda d: d["layers"][0]["mixer"].update(kv_heads=3))
    broken(lambda d: d["layers"][0]["mixer"].pop("conv"))
    broken(lambda d: d["layers"][1]["mixer"]["rot"].update(dims=12))       # more than a head holds
    broken(lambda d: d["layers"][1]["mixer"]["rot"].update(dims=3))
    broken(lambda d: d["layers"][1]["mixer"]["mask"].update(size=0))
    broken(lambda d: d["layers"][1]["mixer"]["mask"].update(keep_first=-1))
    broken(lambda d: d["layers"][1]["mixer"].pop("scale"))
    broken(lambda d: d["layers"][2]["mixer"].update(rot_dim=8))            # rot.dims is rot_dim
    broken(lambda d: d["layers"][2]["mixer"].pop("kv_rank"))
    broken(lambda d: d["layers"][1]["mlp"].update(kind="gelu"))
    broken(lambda d: d["layers"][1]["mlp"].pop("ff"))
    broken(lambda d: d["layers"][0]["mlp"]["router"].update(top=7))        # the kept groups hold six
    broken(lambda d: d["layers"][0]["mlp"]["router"].update(identity=1))   # eight in three groups
    broken(lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(keep=4))
    broken(lambda d: d.update(logit_softcap=0.0))
    broken(lambda d: d["token_side"].pop("dim"))
    broken(lambda d: d.pop("residual_mult"))
    broken(lambda d: d.pop("norm"))
    broken(lambda d: d.update(layers=[]))


def test_declared_tensors():
    from airframe_b200.config import config_from_dict
    from airframe_b200.engine.model import declared_weights
    got = declared_weights(config_from_dict(RA).model_spec())
    decls = {d.name: tuple(d.shape) for d in got}
    assert len(decls) == len(got)
    assert decls["embed"] == (211, 72) and decls["head"] == (211, 72) and decls["side.embed"] == (211, 60)
    assert decls["final.norm"] == (72,) and decls["final.norm.b"] == (72,)
    assert decls["l0.mix.q"] == (24, 72) and decls["l0.mix.v"] == (80, 72) and decls["l0.mix.v.conv"] == (80, 3)
    assert decls["l0.mix.b"] == (4, 72) and decls["l0.mix.A_log"] == (4,) and decls["l0.mix.dt_bias"] == (48,)
    assert decls["l0.mix.a1"] == (10, 72) and decls["l0.mix.a2"] == (48, 10) and decls["l0.mix.g2"] == (80, 10)
    assert decls["l4.mix.g1"] == (13, 72) and decls["l4.mix.a1"] == (7, 72) and decls["l0.mix.norm"] == (20,)
    assert decls["l1.mix.q.norm"] == (60,) and decls["l1.mix.k.norm"] == (30,) and decls["l1.mix.o"] == (72, 84)
    assert decls["l2.mix.g"] == (42, 72) and decls["l2.mix.dkv"] == (26, 72) and decls["l2.mix.q"] == (48, 72)
    assert decls["l0.mlp.router"] == (9, 72) and decls["l0.mlp.correction"] == (9,) and decls["l0.mlp.e6.down"] == (72, 28)
    assert "l0.mlp.e7.up" not in decls and "l2.norm2" not in decls and decls["l1.mlp.up"] == (52, 72)
    assert decls["l2.side.gate"] == (12, 72) and decls["l2.side.proj"] == (72, 12) and decls["l2.side.norm"] == (72,)
    assert not any("side" in d.name for d in declared_weights(config_from_dict(RC).model_spec()))


def test_ranks_that_only_the_tensors_give(tmp_path):
    """A folder whose config.json does not say the low ranks loads all the same (they are read from the tensors)."""
    from airframe_b200.config import config_from_folder
    from airframe_b200.engine.model import declared_weights
    folder = make_folder(RC, seed=1, root=tmp_path)
    d = json.loads((folder / "config.json").read_text())
    for layer in d["layers"]:
        layer["mixer"].pop("rank", None)
    (folder / "config.json").write_text(json.dumps(d))
    from airframe_b200.weights.loader import SafetensorsFolder, load_weights
    got = load_weights(SafetensorsFolder(folder), declared_weights(config_from_folder(folder).model_spec()), torch.float32, "cpu")
    assert tuple(got["l0.mix.a1"].shape) == (5, 50)


def test_what_a_layer_keeps_per_sequence():
    """A delta layer keeps its heads' states and the convolutions' last inputs (no convolution: the states alone); a window
    with kept tokens keeps their pages and the ring's; freed slots come back zeroed."""
    from airframe_b200.cache import SequenceCache
    from airframe_b200.config import config_from_dict
    from airframe_b200.engine import Model
    needs = Model(config_from_dict(RA).model_spec(), torch.float32, "cpu").cache_needs()
    assert all(n[2] is None and n[3] is None for n in needs)
    assert [s.shape for s in needs[0][1]] == [(4, 20, 12), (2, 128)] and [s.shape for s in needs[4][1]] == [(3, 6, 10), (4, 78)]
    assert [n[0] is not None for n in needs] == [False, True, True, True, False]
    assert [s.shape for s in Model(config_from_dict(RC).model_spec(), torch.float32, "cpu").cache_needs()[0][1]] == [(3, 6, 10)]
    c = SequenceCache(needs, 1024, 512, torch.float32, "cpu", max_sequences=3)
    assert c.views[1].kv.ring_rows == 64 and c.views[1].kv.keep_first == 3 and c.views[1].kv.page_table.shape[1] == 2
    assert c.views[3].kv.ring_rows == 128 and c.views[3].kv.keep_first == 67 and c.views[3].kv.page_table.shape[1] == 4
    assert c.views[2].kv.ring_rows == 0 and c.views[2].kv.page_table.shape[1] == 8
    s = c.take_slot()
    for v in (c.views[0], c.views[4]):
        for t in v.state:
            t[s] = 5.0
    c.reserve({s: 500})
    assert sorted(c.pages_held().values()) == [2, 4, 8]          # kept page + ring page; two kept + two; every page
    c.free_slot(s)
    assert set(c.pages_held().values()) == {0}
    again = [c.take_slot() for _ in range(3)]
    assert s in again and all(float(t.abs().max()) == 0 for v in (c.views[0], c.views[4]) for t in v.state)


def test_pages_of_a_window_that_keeps_first_tokens():
    """Pages are taken one by one as a sequence grows, up to the kept ones and the ring, and no more."""
    from airframe_b200.cache.sequence_cache import KVGroup
    from airframe_b200.parts.base import KVNeed
    g = KVGroup(KVNeed(1, 8, 100, keep_first=65), [0], 2, 12, 4096, torch.float32, None)
    assert (g.kept_rows, g.ring_rows, g.pages_per_seq) == (128, 128, 4)
    for n, pages in ((1, 1), (64, 1), (65, 2), (128, 2), (129, 3), (192, 3), (193, 4), (256, 4), (257, 4), (3000, 4)):
        g.grow(0, n)
        assert len(g.held[0]) == pages, n
    assert g.room(0) > 1 << 40
    g.release(0)
    assert g.pages.n_held == 0
    short = KVGroup(KVNeed(1, 8, 100, keep_first=65), [0], 2, 12, 150, torch.float32, None)
    assert short.pages_per_seq == 3                               # (no sequence grows beyond the context)


# ---------------------------------------------------------------- the plain implementation on cases known by hand

def test_plain_window_with_kept_tokens():
    m = plain.visible(7, 2, 3)
    assert m[6].tolist() == [True, True, True, False, False, True, True]
    assert m[3].tolist() == [True, True, True, True, False, False, False] and m[1].tolist() == [True, True] + [False] * 5
    assert plain.visible(4, None, 0).tolist() == torch.ones(4, 4).tril().bool().tolist()
    q = torch.zeros(3, 1, 1, dtype=F64)
    v = torch.tensor([[[1.0]], [[10.0]], [[100.0]]], dtype=F64)
    assert torch.allclose(plain.attend(q, q, v, 1.0, plain.visible(3, 1, 1))[:, 0], torch.tensor([1.0, 5.5, 50.5], dtype=F64))


def test_plain_delta_rule_by_hand():
    w = torch.tensor([[0.5, 2.0], [1.0, 0.0]], dtype=F64)
    x = torch.tensor([[1.0, 1.0], [3.0, 5.0]], dtype=F64)
    assert plain.short_conv(x, w).tolist() == [[2.0, 0.0], [6.5, 1.0]]       # channel 1 sees the token before only
    u = plain.unit(torch.tensor([[3.0, 4.0]], dtype=F64))
    assert torch.allclose(u, torch.tensor([[0.6, 0.8]], dtype=F64), atol=1e-7)
    k = torch.tensor([[1.0, 0.0], [1.0, 0.0]], dtype=F64)
    v = torch.tensor([[4.0], [10.0]], dtype=F64)
    g = torch.tensor([[1.0, 1.0], [0.5, 1.0]], dtype=F64)
    # the first write leaves 0.5 * 4 = 2; it decays to 1; the second moves it by 0.25 (10 - 1)
    assert plain.delta_scan(k, k, v, g, torch.tensor([0.5, 0.25], dtype=F64))[:, 0].tolist() == [2.0, 3.25]
    W = {"a1": torch.zeros(1, 1, dtype=F64), "a2": torch.zeros(2, 1, dtype=F64), "dt_bias": torch.tensor([0.0, -50.0], dtype=F64),
         "A_log": torch.tensor([math.log(3.0)], dtype=F64)}
    d = plain.channel_decay(torch.ones(1, 1, dtype=F64), W, "", 1, 2)
    assert abs(float(d[0, 0, 0]) - 0.125) < 1e-12 and abs(float(d[0, 0, 1]) - 1.0) < 1e-12      # exp(-3 ln 2), and nothing forgotten


def test_plain_choice_groups_and_identity():
    s = torch.tensor([0.4, 0.1, 0.3, 0.2], dtype=F64)
    zero = torch.zeros(4, dtype=F64)
    assert plain.choose(s, zero, 2, 1, 1) == [0, 2]
    assert plain.choose(s, zero, 2, 2, 1) == [0, 1]                          # the group with the largest score, not the largest sum
    # every choice score negative: what is not in a kept group is out, not zero
    assert plain.choose(s, torch.tensor([-1.0, -1.0, -0.5, -2.0], dtype=F64), 2, 2, 1) == [2, 3]
    W = {"m.router": torch.tensor([[0.0], [0.0]], dtype=F64), "m.correction": torch.tensor([0.0, 1.0], dtype=F64),
         "m.e0.gate": torch.tensor([[1.0]], dtype=F64), "m.e0.up": torch.tensor([[2.0]], dtype=F64), "m.e0.down": torch.tensor([[3.0]], dtype=F64)}
    h = torch.tensor([[1.0]], dtype=F64)
    out = plain.experts(h, W, "m.", {"router": {"experts": 1, "identity": 1, "top": 1}})
    assert float(out) == 0.5                                                 # the identity expert, weighted by its score without the correction
    W["m.correction"] = torch.zeros(2, dtype=F64)
    both = plain.experts(h, W, "m.", {"router": {"experts": 1, "identity": 1, "top": 2}})
    assert abs(float(both) - 0.5 * (6.0 / (1.0 + math.exp(-1.0)) + 1.0)) < 1e-12


# ---------------------------------------------------------------- the engine

gpu = pytest.mark.gpu


@pytest.fixture(params=["float32", "bfloat16"])
def dtype(request):
    return request.param


_CASES = {}


def rms_rel(got, ref) -> float:
    d = got.double().cpu() - ref.double()
    return float(d.pow(2).mean().sqrt() / ref.double().pow(2).mean().sqrt())


class Ref:
    """Reference logits, and how far they move (root mean square against theirs) when nothing but every sublayer's
    input is rounded to bfloat16: the least that any bfloat16 computation of them must show."""
    def __init__(self, logits, noise=0.0):
        self.logits, self.noise = logits, noise

    def __getitem__(self, k):
        return Ref(self.logits[k], self.noise)


def agrees(got, ref, dtype, what=None):
    """32-bit: the largest difference against the largest reference logit.  bfloat16: position by position, the root mean
    square of the differences against that of all logits: half the positions within 3e-2 and all within 8e-2 (or three
    and eight times what rounding the sublayers' inputs alone does to the plain logits, where that is more), but for the few
    (two, or one in ten) whose choice of experts rests on a call so close that rounding decides it."""
    if dtype == "float32":
        assert rel_err(got, ref.logits) < VS_PLAIN[dtype], what
        return
    d = (got.double().cpu() - ref.logits.double()).pow(2).mean(-1).sqrt() / ref.logits.double().pow(2).mean().sqrt()
    assert float(d.median()) < max(3e-2, 3.0 * ref.noise), (what, float(d.median()))
    over = int((d > max(8e-2, 8.0 * ref.noise)).sum())
    assert over <= max(2, d.numel() // 10), (what, over, d.numel(), float(d.max()))


def case(name, tmp_path_factory, edit=None, key=None, cfg_edit=None):
    key = key or name
    if key not in _CASES:
        cfg_dict = copy.deepcopy(CONFIGS[name])
        if cfg_edit is not None:
            cfg_edit(cfg_dict)
        folder = make_folder(cfg_dict, seed=71 + len(_CASES), root=tmp_path_factory.mktemp("rd" + key), edit=edit)
        cfg, w = plain.read_model_folder(folder)
        _CASES[key] = {"folder": folder, "cfg": cfg, "w": w, "ref": {}}
    return _CASES[key]


def reference(c, ids):
    k = tuple(ids)
    if k not in c["ref"]:
        exact = plain.logits(c["cfg"], c["w"], ids)
        rounded = plain.forward(c["cfg"], c["w"], ids, round_h=lambda z: z.to(torch.bfloat16).to(F64))
        c["ref"][k] = Ref(exact, rms_rel(rounded, exact))
    return c["ref"][k]


def load(c, dtype, max_tokens=64 * 24, **kw):
    from airframe_b200.engine import GpuRuntime
    return GpuRuntime.load(c["folder"], dtype=dtype, max_tokens=max_tokens, **kw)


@gpu
@pytest.mark.parametrize("name", ["A", "B", "C", "D", "E"])
def test_whole_prompt_and_token_by_token(name, dtype, tmp_path_factory):
    """A prompt in one step; the same tokens with the last 40 one by one (the captured decode step); a prompt of one
    token followed by single tokens only (the convolutions and the states begin at zero); two tokens and a few more."""
    c = case(name, tmp_path_factory)
    rt = load(c, dtype)
    ids = replay.random_ids(c["cfg"]["vocab"], 150, 5)
    ref = reference(c, ids)
    whole = replay.run_whole(rt, ids)
    agrees(whole, ref, dtype)
    tail = replay.run_tail(rt, ids, 40)
    agrees(tail, ref, dtype)
    if dtype == "float32":
        assert rel_err(tail, whole) < SPLITS[dtype] * 4
    agrees(replay.run_tail(rt, ids[:70], 69), ref[:70], dtype)
    agrees(replay.run_whole(rt, ids[:1]), ref[:1], dtype)
    agrees(replay.run_tail(rt, ids[:9], 7), ref[:9], dtype)


@gpu
@pytest.mark.parametrize("name", ["A", "B", "C", "E"])
def test_unequal_batches_and_slots_used_again(name, dtype, tmp_path_factory):
    """Requests of unequal lengths (one of a single token) in batches, then decoded together, the shorter ones leaving;
    twice, so that slots, their states, rows and pages are used again by other requests."""
    c = case(name, tmp_path_factory)
    rt = load(c, dtype)
    V = c["cfg"]["vocab"]
    reqs = [replay.random_ids(V, n, 100 + n) for n in (90, 1, 37, 160, 66, 12)]
    refs = [reference(c, r) for r in reqs]
    prompt_lens = [70, 1, 5, 150, 64, 2]
    seen = []
    for rnd in range(2):
        out, slots = replay.run_batches(rt, reqs, 4, prompt_lens)
        seen.append(slots)
        for i, r in enumerate(refs):
            agrees(out[i], r, dtype, (rnd, i))
    assert seen[0] == seen[1]
    alone = replay.run_tail(rt, reqs[3], 10)
    if dtype == "float32":
        assert rel_err(alone, out[3]) < SPLITS[dtype] * 4
    else:
        agrees(alone, refs[3], dtype)
    # prompts of one token each, several at a time: a prefill step of single tokens
    out, _ = replay.run_batches(rt, [r[:6] for r in reqs if len(r) > 6], 5, [1] * 5)
    for i, r in enumerate(r for r in refs if r.logits.shape[0] > 6):
        agrees(out[i], r[:6], dtype, i)


@gpu
@pytest.mark.parametrize("name", ["A", "B", "E"])
def test_long_decoding_over_pages(name, dtype, tmp_path_factory):
    """Three tokens of prompt, then 290 single tokens: cache pages begin at 64, 128, 192 and 256, states and rows are
    carried 290 times, rings wrap around beside their kept pages."""
    c = case(name, tmp_path_factory)
    rt = load(c, dtype)
    ids = replay.random_ids(c["cfg"]["vocab"], 293, 9)
    tail = replay.run_tail(rt, ids, 290)
    agrees(tail, reference(c, ids), dtype)
    whole = replay.run_whole(rt, ids)
    agrees(whole, reference(c, ids), dtype)
    if dtype == "float32":
        assert rms_rel(tail, whole.double()) < 1e-5


@gpu
@pytest.mark.parametrize("name", ["A", "B"])
def test_long_prompts_in_chunks(name, dtype, tmp_path_factory):
    """Prompts of five and a half chunks and of four chunks and one token: alone, with their last tokens one by one (the
    states the chunks left), and both beside a short request in one step."""
    c = case(name, tmp_path_factory)
    rt = load(c, dtype, max_tokens=64 * 40)
    V = c["cfg"]["vocab"]
    reqs = [replay.random_ids(V, n, 500 + n) for n in (700, 513, 5)]
    refs = [reference(c, r) for r in reqs]
    agrees(replay.run_whole(rt, reqs[0]), refs[0], dtype)
    agrees(replay.run_tail(rt, reqs[0], 30), refs[0], dtype)
    out, _ = replay.run_batches(rt, reqs, 3, [690, 513, 3])
    for i, r in enumerate(refs):
        agrees(out[i], r, dtype, i)


def _loud(name, t):
    """Token 0's embedding made large, and queries and keys scaled up: what one position leaves in keys and states is then
    seen from far away."""
    if name == "embed":
        t = t.clone()
        t[0] *= 5.0
    if name.endswith(("mix.q.norm", "mix.k.norm")):
        t = t * 1.7
    return t


@gpu
@pytest.mark.parametrize("name", ["A", "B", "E"])
@pytest.mark.parametrize("at", [0, 4, 63, 64])
def test_far_tokens_show(name, at, dtype, tmp_path_factory):
    """A loud token (the first, one inside the kept tokens or right behind them, the last row of a cache page, the first of
    the next) reaches the last logits some 250 positions on: the plain logits move far beyond the tolerance without it, and
    the engine's agree with it."""
    c = case(name, tmp_path_factory, key=name + "-far", edit=_loud)
    cfg, w = c["cfg"], c["w"]
    ids = [i + 1 for i in replay.random_ids(cfg["vocab"] - 1, 250 + at, 33)]
    ids[at] = 0
    ref = reference(c, ids)
    other = list(ids)
    other[at] = 1
    assert rel_err(plain.logits(cfg, w, other)[-8:], ref.logits[-8:]) > 10 * VS_PLAIN["float32"]
    rt = load(c, dtype)
    agrees(replay.run_tail(rt, ids, 8)[-8:], ref[-8:], dtype)
    agrees(replay.run_whole(rt, ids)[-8:], ref[-8:], dtype)
    agrees(replay.run_tail(rt, ids, 200)[-8:], ref[-8:], dtype)


@gpu
@pytest.mark.parametrize("size,keep", [(1, 0), (5, 1), (64, 64), (63, 65), (65, 63), (128, 130), (200, 10)])
@pytest.mark.parametrize("dim", [64, 128, 24])
def test_window_edges_against_kept_tokens(size, keep, dim, dtype, tmp_path_factory):
    """One attention layer (heads of 64, 128 and an odd size: every kernel) with windows and kept tokens at, just inside and
    just outside page borders: a prompt, and decoding over more than the ring, at every position."""
    layer = {"type": "attention", "mlp": None, "mixer": {
        "heads": 4, "kv_heads": 2, "dim": dim, "vdim": dim, "scale": 0.3, "rot": {"base": 100.0, "dims": 8},
        "mask": {"size": size, "keep_first": keep}}}
    cfg = {"architecture": "Retudra", "vocab": 64, "width": 64, "norm": {"eps": 1e-5}, "residual_mult": 1.0, "logit_softcap": None,
           "token_side": None, "layers": [layer]}
    folder = make_folder(cfg, seed=size + keep + dim, root=tmp_path_factory.mktemp("win"), edit=_loud)
    got_cfg, w = plain.read_model_folder(folder)
    c = {"folder": folder, "cfg": got_cfg, "w": w, "ref": {}}
    ids = replay.random_ids(64, 420, size * 7 + keep)
    ref = reference(c, ids)
    rt = load(c, dtype)
    agrees(replay.run_whole(rt, ids), ref, dtype)
    agrees(replay.run_tail(rt, ids, 330), ref, dtype)
    a, b = ids[:300], ids[100:170]
    out, _ = replay.run_batches(rt, [a, b, a], 3, [100, 60, 290])
    agrees(out[0], ref[:300], dtype)
    agrees(out[1], reference(c, b), dtype)
    agrees(out[2], ref[:300], dtype)


@gpu
def test_what_a_mechanism_left_out_would_do(dtype, tmp_path_factory):
    """Leaving out the convolution, the step sizes, the decay, a gate, a norm's weights or bias, the kept tokens, one position
    of a window, a rotation, the correction, the groups, the identity experts, the side input, the softcap or the residual
    factor moves the plain logits far beyond the tolerance that the engine keeps."""
    c = case("A", tmp_path_factory)
    cfg, w = c["cfg"], c["w"]
    ids = replay.random_ids(cfg["vocab"], 150, 8)
    ref = reference(c, ids)

    def moved(w2=None, cfg2=None):
        return rms_rel(plain.logits(cfg2 or cfg, w2 or w, ids), ref.logits)

    def weights(change, *ends):
        return {k: (change(v) if k.endswith(ends) else v) for k, v in w.items()}

    def changed(edit):
        d = copy.deepcopy(cfg)
        edit(d)
        return d

    def last_tap(v):
        v = torch.zeros_like(v)
        v[:, -1] = 1.0
        return v

    least = 10 * VS_PLAIN["float32"]
    zero, one = torch.zeros_like, torch.ones_like
    assert moved(weights(last_tap, ".conv")) > 0.01
    assert moved(weights(zero, ".mix.b")) > least
    assert moved(weights(lambda v: v - 50.0, ".dt_bias")) > 0.01              # nothing decays
    assert moved(weights(zero, ".a2")) > least
    assert moved(weights(zero, ".A_log")) > least
    assert moved(weights(zero, "l0.mix.g1")) > least
    assert moved(weights(zero, "l2.mix.g")) > least
    assert moved(weights(one, "l1.mix.q.norm", "l3.mix.k.norm", ".dkv.norm", "l0.mix.norm")) > least
    assert moved(weights(zero, ".norm1.b", ".norm2.b")) > 0.01
    assert moved(weights(zero, ".correction")) > least
    assert moved(weights(zero, "side.embed")) > 0.01
    assert moved(cfg2=changed(lambda d: d["layers"][1]["mixer"]["mask"].update(keep_first=0))) > least
    assert moved(cfg2=changed(lambda d: d["layers"][1]["mixer"]["mask"].update(keep_first=2))) > least
    assert moved(cfg2=changed(lambda d: d["layers"][3]["mixer"]["mask"].update(keep_first=66))) > least
    assert moved(cfg2=changed(lambda d: d["layers"][1]["mixer"]["mask"].update(size=10))) > least
    assert moved(cfg2=changed(lambda d: d["layers"][3]["mixer"]["mask"].update(size=69))) > least
    assert moved(cfg2=changed(lambda d: d["layers"][1]["mixer"]["rot"].update(dims=0))) > least
    assert moved(cfg2=changed(lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(keep=3))) > least
    assert moved(cfg2=changed(lambda d: d.update(residual_mult=1.0))) > 0.01
    assert moved(cfg2=changed(lambda d: d.update(logit_softcap=None))) > 0.01
    rt = load(c, dtype)
    agrees(replay.run_whole(rt, ids), ref, dtype)
    agrees(replay.run_tail(rt, ids, 85), ref, dtype)


@gpu
def test_layers_agree_one_by_one(tmp_path_factory):
    """The residual stream after every run of a layer, 32-bit, against the plain implementation's."""
    from airframe_b200.engine import StepEntry

    class Keep:
        def __init__(self):
            self.x = []

        def after(self, run, layer, x, batch):
            if run >= 0:
                self.x.append(x.detach().cpu().double())

    for name in CONFIGS:
        c = case(name, tmp_path_factory)
        rt = load(c, "float32")
        ids = replay.random_ids(c["cfg"]["vocab"], 75, 2)
        per_layer = []
        plain.forward(c["cfg"], c["w"], ids, layers_out=per_layer)
        s = rt.engine.take_slot()
        keep = Keep()
        rt.engine.step([StepEntry(s, ids, [0])], probe=keep)
        rt.engine.free_slot(s)
        assert len(keep.x) == len(per_layer)
        for i, (got, ref) in enumerate(zip(keep.x, per_layer)):
            assert rel_err(got, ref) < 2e-5, (name, i)


@gpu
def test_greedy_generation_through_the_runtime(tmp_path_factory):
    from airframe_b200.sampling import SamplingParams
    for name in ("A", "D"):
        c = case(name, tmp_path_factory)
        rt = load(c, "float32")
        V = c["cfg"]["vocab"]
        prompts = [replay.random_ids(V, n, 60 + n) for n in (9, 1, 30)]
        params = SamplingParams(max_tokens=12, temperature=0.0, repetition_penalty=1.0, ignore_eos=True)
        got = rt.generate(prompts, params)
        want = [plain.generate_greedy(c["cfg"], c["w"], p, 12) for p in prompts]
        assert got == want
        assert rt.generate(prompts[2], params) == want[2]
        rt16 = load(c, "bfloat16")
        assert [len(o) for o in rt16.generate(prompts, params)] == [12, 12, 12]


@gpu
def test_trace_replay_of_a_retudra_folder(tmp_path, tmp_path_factory):
    from airframe_b200.cli.trace_run import main
    c = case("C", tmp_path_factory)
    V = c["cfg"]["vocab"]
    a, b = replay.random_ids(V, 20, 1), replay.random_ids(V, 7, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:18], "want": [0, 17]},
                                     {"id": "b", "tokens": b[:6], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [a[18]], "want": [0]},
                                     {"id": "b", "tokens": [b[6]], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": [a[19]], "want": []}], "end": ["a"]}]
    out = io.StringIO()
    code = main(["--model", str(c["folder"]), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "128"],
                stdin=io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"), stdout=out)
    assert code == 0 and out.getvalue().split() == ["done", "0", "done", "1", "done", "2"]
    import numpy as np
    ra, rb = reference(c, a).logits, reference(c, b).logits
    s0 = torch.from_numpy(np.fromfile(tmp_path / "0.f32", dtype="<f4")).view(2, V)
    s1 = torch.from_numpy(np.fromfile(tmp_path / "1.f32", dtype="<f4")).view(2, V)
    assert rel_err(s0, ra[[0, 17]]) < VS_PLAIN["float32"]
    assert rel_err(s1, torch.stack([ra[18], rb[6]])) < VS_PLAIN["float32"]
    assert not (tmp_path / "2.f32").exists()


@gpu
def test_long_prompt_at_layer_sizes_beyond_the_plain_implementation(tmp_path_factory):
    """The named small configuration (tensor-core products, attention, delta rule and experts) on a prompt of 2,500
    tokens, then 70 single tokens: too long for the plain implementation, so the engine is held against itself: the
    32-bit logits must not depend on where the prompt ends and the single tokens begin, and bfloat16 must agree with
    32-bit within its rounding."""
    from airframe_b200.config.presets import preset
    folder = make_folder(preset("retudra-small"), seed=4, root=tmp_path_factory.mktemp("rdsmall"))
    from airframe_b200.engine import GpuRuntime, StepEntry
    ids = replay.random_ids(8192, 2570, 17)
    want = [0, 1, 255, 256, 257, 1023, 2047, 2499]

    def run(dtype, cut):
        rt = GpuRuntime.load(folder, dtype=dtype, max_tokens=64 * 48, max_context=4096)
        s = rt.engine.take_slot()
        out = [rt.step([StepEntry(s, ids[:cut], [w for w in want if w < cut])]).cpu()]
        for t in ids[cut:]:
            out.append(rt.step([StepEntry(s, [t], [0])]).cpu())
        rt.engine.free_slot(s)
        return torch.cat(out)

    a = run("float32", 2500)
    assert torch.isfinite(a).all()
    b = run("float32", 2540)
    assert rel_err(b[-30:], a[-30:]) < 1e-4
    c = run("bfloat16", 2500)
    assert rms_rel(c, a) < 6e-2
