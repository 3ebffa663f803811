"""Teselix through the engine against the plain implementation (``plain_teselix``): every way of
cutting the same requests into steps, in 32-bit and bfloat16, on configurations that differ in every
size, in the order of their layers, in which layers share weights and in their constants."""
import copy
import io
import json
import math

import pytest
import torch

import plain_teselix as plain
import replay
from tiny_teselix import CONFIGS, TA, TB, TC, make_folder
from tolerances import SPLITS, VS_PLAIN, rel_err

F64 = torch.float64


# ---------------------------------------------------------------- configuration (no GPU)

def test_config_round_trip_and_registry():
    from airframe_b200.config import TeselixConfig, config_from_dict
    cfg = config_from_dict(TA)
    assert isinstance(cfg, TeselixConfig)
    assert config_from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg
    spec = cfg.model_spec()
    # three layers have weights of their own; the others run them again with a cache and states of their own
    assert [layer.prefix for layer in spec.layers] == ["l0.", "l1.", "l3."]
    assert [e.layer for e in spec.schedule] == [0, 1, 1, 2, 0, 1]
    assert all(e.cache_from is None and e.enter is None for e in spec.schedule)
    assert [(layer.block.kind, layer.mixer.kind, layer.feed_forward.kind) for layer in spec.layers] == \
        [("normed_sum", "retention", "routed_experts"), ("normed_sum", "latent_attention", "routed_experts"),
         ("normed_sum", "retention", "none")]
    block = spec.layers[1].block.params
    assert (block["alpha"], block["shift_weight"]) == (1.7, "l1.shift")
    assert block["gates"] == [{"weight": "l1.rg1", "bias": "l1.rg1.b"}, {"weight": "l1.rg2", "bias": "l1.rg2.b"}]
    assert spec.layers[0].norms["mixer_sum"].params == {"weight": "l0.norm1", "bias": "l0.norm1.b", "size": 72, "eps": 1e-5}
    assert spec.layers[2].norms.keys() == {"mixer_sum"}
    ret = spec.layers[0].mixer.params
    assert (ret["num_heads"], ret["head_dim"], ret["value_dim"], ret["decay"]) == (2, 12, 20, [0.9, 0.97])
    assert (ret["position"].params["pairing"], ret["position"].params["rotary_dim"], ret["position"].params["theta"]) == ("half", 8, 50.0)
    lat = spec.layers[1].mixer.params
    assert (lat["num_heads"], lat["head_dim"], lat["rot_dim"], lat["value_dim"], lat["kv_rank"], lat["q_rank"]) == (3, 10, 6, 14, 20, 18)
    assert lat["window"] is None and lat["scale"] == 0.3 and lat["position"].params["pairing"] == "adjacent"
    assert lat["position"].params["scaling"] == {"factor": 3.0, "original": 40.0, "fast": 8.0, "slow": 0.5}
    ff = spec.layers[0].feed_forward.params
    assert (ff["num_experts"], ff["top"], ff["limit"], ff["intermediate_size"], ff["vocab_size"]) == (5, 2, 1.5, 36, 211)
    assert ff["table_weight"] == "l0.mlp.table" and ff["shared"]["limit"] == 0.8 and "router_weight" not in ff
    assert "shared" not in config_from_dict(TC).model_spec().layers[1].feed_forward.params
    assert spec.head.params["tied_to"] == "embed" and spec.final_norm.params["bias"] == "final.norm.b"


def test_config_refuses_what_it_does_not_know():
    from airframe_b200.config import ConfigError, config_from_dict

    def broken(edit):
        d = copy.deepcopy(TA)
        edit(d)
        with pytest.raises(ConfigError):
            config_from_dict(d)

    broken(lambda d: d["layers"][3].update(type="gla"))
    broken(lambda d: d["layers"][3]["mixer"].update(decay=[0.5, 0.8]))
    broken(lambda d: d["layers"][3]["mixer"].pop("decay"))
    broken(lambda d: d["layers"][3]["mixer"]["rot"].update(dims=12))       # more than a head holds
    broken(lambda d: d["layers"][3]["mixer"]["rot"].update(dims=3))
    broken(lambda d: d["layers"][1]["mixer"].update(rot_dim=8))            # rot.dims is rot_dim
    broken(lambda d: d["layers"][1]["mixer"].pop("q_rank"))
    broken(lambda d: d["layers"][1]["mixer"].pop("scale"))
    broken(lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"))
    broken(lambda d: d["layers"][0]["mlp"].update(kind="dense"))
    broken(lambda d: d["layers"][0]["mlp"]["router"].update(top=6))
    broken(lambda d: d["layers"][0]["mlp"]["expert"].pop("limit"))
    broken(lambda d: d["layers"][0]["mlp"]["shared"].pop("ff"))
    broken(lambda d: d["layers"][4].update(weights_of=9))
    broken(lambda d: d["layers"][4].update(weights_of=4))
    broken(lambda d: (d["layers"][0].update(weights_of=4)))                # a circle
    broken(lambda d: d["layers"][4].update(weights_of=3))                  # another kind of sizes
    broken(lambda d: d.pop("postln_alpha"))
    broken(lambda d: d.pop("norm"))
    broken(lambda d: d.update(layers=[]))


def test_declared_tensors():
    from airframe_b200.config import config_from_dict
    from airframe_b200.engine.model import declared_weights
    got = declared_weights(config_from_dict(TA).model_spec())
    decls = {d.name: tuple(d.shape) for d in got}
    assert len(decls) == len(got)
    assert decls["embed"] == (211, 72) and decls["final.norm"] == (72,) and decls["final.norm.b"] == (72,) and "head" not in decls
    assert decls["l0.mix.q"] == (24, 72) and decls["l0.mix.v"] == (40, 72) and decls["l0.mix.g"] == (40, 72) and decls["l0.mix.o"] == (72, 40)
    assert decls["l1.mix.dq"] == (18, 72) and decls["l1.mix.dq.norm"] == (18,) and decls["l1.mix.uq"] == (48, 18)
    assert decls["l1.mix.dkv"] == (26, 72) and decls["l1.mix.uk"] == (30, 20) and decls["l1.mix.uv"] == (42, 20)
    assert decls["l1.mix.sink"] == (3,) and decls["l1.mix.g"] == (3, 72) and decls["l1.mix.o"] == (72, 42)
    assert decls["l0.mlp.table"] == (211, 2) and decls["l1.mlp.table"] == (211, 1) and decls["l0.mlp.e4.gate"] == (36, 72)
    assert decls["l0.mlp.shared.down"] == (72, 40) and "l0.mlp.e5.gate" not in decls
    assert decls["l0.rg1"] == (72, 72) and decls["l0.rg2.b"] == (72,) and decls["l0.shift"] == (72,) and decls["l3.norm1.b"] == (72,)
    assert not any(n.startswith(("l2.", "l4.", "l5.")) for n in decls) and "l3.norm2" not in decls and "l3.rg2" not in decls
    table = next(d for d in got if d.name == "l0.mlp.table")
    assert (table.kind, table.below) == ("choice_table", 5)
    from airframe_b200.weights.random_init import RandomSource
    t = RandomSource(got, 3).read("l0.mlp.table")
    assert t.dtype == torch.int32 and int(t.min()) >= 0 and int(t.max()) < 5 and bool((t[:, 0] != t[:, 1]).all())


def test_what_a_layer_keeps_per_sequence():
    """Every run has a shift's row of its own beside its mixer's state or cached rows; freed slots come back zeroed."""
    from airframe_b200.cache import SequenceCache
    from airframe_b200.config import config_from_dict
    from airframe_b200.engine import Model
    needs = Model(config_from_dict(TA).model_spec(), torch.float32, "cpu").cache_needs()
    assert [n[3].shape for n in needs] == [(72,)] * 6 and all(n[2] is None for n in needs)
    assert [n[1].shape if n[1] else None for n in needs] == [(2, 20, 12), None, None, (3, 6, 10), (2, 20, 12), None]
    assert [n[0] is not None for n in needs] == [False, True, True, False, False, True]
    c = SequenceCache(needs, 640, 256, torch.float32, "cpu", max_sequences=3)
    views = c.views
    assert len({v.block_state.data_ptr() for v in views}) == 6
    assert len({v.kv.k.data_ptr() for v in views if v.kv is not None}) == 3
    s = c.take_slot()
    for v in views:
        v.block_state[s] = 5.0
        if v.state is not None:
            v.state[s] = 5.0
    c.free_slot(s)
    again = [c.take_slot() for _ in range(3)]
    assert s in again
    assert all(float(v.block_state.abs().max()) == 0 and (v.state is None or float(v.state.abs().max()) == 0) for v in views)


# ---------------------------------------------------------------- the plain implementation on cases known by hand

def test_plain_norm_gate_and_shift():
    x = torch.tensor([[1.0, 3.0]], dtype=F64)
    y = plain.layer_norm(x, torch.tensor([2.0, 10.0], dtype=F64), torch.tensor([0.5, 0.0], dtype=F64), 3.0)
    assert y.tolist() == [[2.0 * -0.5 + 0.5, 10.0 * 0.5]]                   # mean 2, variance 1, root of 1 + 3
    s = plain.norm_of_sum(x, torch.tensor([[1.0, 1.0]], dtype=F64), 2.0, torch.ones(2, dtype=F64), torch.zeros(2, dtype=F64), 0.0)
    assert s.tolist() == [[-1.0, 1.0]]                                      # 2 * [1, 3] + 1 = [3, 7]
    g = plain.residual_gate(x, torch.tensor([[1.0, 0.0], [0.0, 0.0]], dtype=F64), torch.tensor([-1.0, 50.0], dtype=F64))
    assert abs(float(g[0, 0]) - 0.5) < 1e-15 and abs(float(g[0, 1]) - 1.0) < 1e-15
    h = torch.tensor([[1.0, 1.0], [5.0, 5.0], [9.0, 9.0]], dtype=F64)
    assert plain.shifted(h, torch.tensor([0.25, 1.0], dtype=F64)).tolist() == [[0.75, 0.0], [4.0, 1.0], [8.0, 5.0]]


def test_plain_rotation_and_stretch():
    f, mag = plain.frequencies({"base": 100.0, "dims": 4})
    assert f.tolist() == [1.0, 0.1] and mag == 1.0
    x = torch.zeros(2, 1, 6, dtype=F64)
    x[1, 0] = torch.tensor([1.0, 2.0, 3.0, 4.0, 5.0, 6.0])
    c1, s1, c2, s2 = math.cos(1.0), math.sin(1.0), math.cos(0.1), math.sin(0.1)
    half = plain.rotate_half_split(x, f, 2.0)[1, 0]
    assert torch.allclose(half, torch.tensor([2 * (c1 - 3 * s1), 2 * (2 * c2 - 4 * s2), 2 * (3 * c1 + s1), 2 * (4 * c2 + 2 * s2), 5.0, 6.0], dtype=F64))
    near = plain.rotate_neighbours(x, f, 1.0)[1, 0]
    assert torch.allclose(near, torch.tensor([c1 - 2 * s1, 2 * c1 + s1, 3 * c2 - 4 * s2, 4 * c2 + 3 * s2, 5.0, 6.0], dtype=F64))
    # pairs that turn often keep their frequency, those that turn rarely are divided by the factor
    sc = {"factor": 4.0, "original": 1000.0, "fast": 32.0, "slow": 1.0}
    f, mag = plain.frequencies({"base": 10000.0, "dims": 32, "scaling": sc})
    plain_f, _ = plain.frequencies({"base": 10000.0, "dims": 32})
    assert abs(mag - (0.1 * math.log(4.0) + 1.0)) < 1e-15
    lo = math.floor(32 * math.log(1000.0 / (2 * math.pi * 32.0)) / (2 * math.log(10000.0)))
    hi = math.ceil(32 * math.log(1000.0 / (2 * math.pi)) / (2 * math.log(10000.0)))
    assert torch.equal(f[:lo + 1], plain_f[:lo + 1]) and torch.allclose(f[hi:], plain_f[hi:] / 4.0)
    r = 1.0 / (hi - lo)
    assert abs(float(f[lo + 1] / plain_f[lo + 1]) - (r / 4.0 + 1.0 - r)) < 1e-12


def test_plain_scan_sink_and_experts():
    q = torch.tensor([[1.0], [1.0], [2.0]], dtype=F64)
    v = torch.tensor([[1.0], [10.0], [100.0]], dtype=F64)
    assert plain.decayed_scan(q, q, v, 0.5)[:, 0].tolist() == [1.0, 10.5, 2.0 * (0.25 + 5.0 + 200.0)]
    p = plain.sink_softmax(torch.zeros(2, 2, dtype=F64), torch.tensor(math.log(2.0), dtype=F64))
    assert torch.allclose(p, torch.tensor([[1 / 3, 0.0], [0.25, 0.25]], dtype=F64))
    W = {"m.e0.gate": torch.tensor([[9.0]], dtype=F64), "m.e0.up": torch.tensor([[-9.0]], dtype=F64), "m.e0.down": torch.tensor([[4.0]], dtype=F64),
         "m.e1.gate": torch.tensor([[0.0]], dtype=F64), "m.e1.up": torch.tensor([[1.0]], dtype=F64), "m.e1.down": torch.tensor([[4.0]], dtype=F64),
         "m.table": torch.tensor([[0, 1], [1, 0]])}
    h = torch.tensor([[1.0]], dtype=F64)
    one = 2.0 / (1.0 + math.exp(-3.404)) * (-2.0 + 1.0) * 4.0                # both limited to 2; the up branch from below
    assert abs(float(plain.clamped_expert(h, W, "m.e0", 2.0)) - one) < 1e-12
    got = plain.table_experts(h, [1], W, "m.", {"router": {"top": 2}, "expert": {"limit": 2.0}})
    assert abs(float(got) - one / 2.0) < 1e-12                               # the second expert's gate is zero
    assert plain.owner(TA["layers"], 5) == 1 and plain.owner(TA["layers"], 4) == 0 and plain.owner(TA["layers"], 3) == 3


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


def agrees(got, ref, dtype, what=None, rms=3e-2, worst=0.15):
    """32-bit: the largest difference against the largest reference logit.  bfloat16: the root mean square of the
    differences against that of the logits, and a looser bound on the largest one; the bounds are ``rms`` and ``worst``,
    or three times what rounding the sublayers' inputs alone does to the plain logits where that is more."""
    if dtype == "float32":
        assert rel_err(got, ref.logits) < VS_PLAIN[dtype], what
        return
    assert rms_rel(got, ref.logits) < max(rms, 3.0 * ref.noise), what
    assert rel_err(got, ref.logits) < max(worst, 12.0 * ref.noise), what


def case(name, tmp_path_factory, edit=None, key=None, cfg_edit=None):
    key = key or name
    if key not in _CASES:
        cfg_dict = copy.deepcopy(CONFIGS[name])
        if cfg_edit is not None:
            cfg_edit(cfg_dict)
        folder = make_folder(cfg_dict, seed=71 + len(_CASES), root=tmp_path_factory.mktemp("tx" + key), edit=edit)
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
    token followed by single tokens only (the shift and the states begin at zero); two tokens and a few more."""
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
@pytest.mark.parametrize("name", ["B", "E"])
def test_long_decoding_over_pages(name, dtype, tmp_path_factory):
    """Three tokens of prompt, then 290 single tokens: cache pages begin at 64, 128, 192 and 256, states and rows are
    carried 290 times, and every key stays visible."""
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
    """Token 0's embedding made large, and what the latent attention attends with scaled up: what one position leaves in
    keys and states is then seen from far away."""
    if name == "embed":
        t = t.clone()
        t[0] *= 5.0
    if name.endswith("mix.uq"):
        t = t * 4.0
    return t


@gpu
@pytest.mark.parametrize("name", ["B", "C"])
@pytest.mark.parametrize("at", [0, 63, 64])
def test_far_tokens_show(name, at, dtype, tmp_path_factory):
    """A loud token (the first, the last row of a cache page, the first of the next) reaches the last logits some 250
    positions on: the plain logits move far beyond the tolerance without it, and the engine's agree with it."""
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
def test_what_a_mechanism_left_out_would_do(dtype, tmp_path_factory):
    """Leaving out the shift, a residual gate, the sinks, the heads' gate, a norm's bias, the limits, the shared expert's
    sum, a rotation, the stretch, the decay or the second factor of the residual sum moves the plain logits far beyond the
    tolerance that the engine keeps."""
    c = case("A", tmp_path_factory)
    cfg, w = c["cfg"], c["w"]
    ids = replay.random_ids(cfg["vocab"], 60, 8)
    ref = reference(c, ids)

    def moved(w2=None, cfg2=None):
        return rms_rel(plain.logits(cfg2 or cfg, w2 or w, ids), ref.logits)

    def weights(change, *ends):
        return {k: (change(v) if k.endswith(ends) else v) for k, v in w.items()}

    def changed(edit):
        d = copy.deepcopy(cfg)
        edit(d)
        return d

    least = 10 * VS_PLAIN["float32"]
    zero = torch.zeros_like
    assert moved(weights(zero, ".shift")) > 0.01
    assert moved(weights(lambda v: torch.full_like(v, 50.0), ".rg1.b")) > 0.01
    assert moved(weights(lambda v: torch.full_like(v, 50.0), ".rg2.b")) > 0.01
    assert moved(weights(lambda v: v - 50.0, ".sink")) > least
    assert moved(weights(zero, "l1.mix.g")) > least
    assert moved(weights(zero, ".norm1.b", ".norm2.b")) > 0.01
    assert moved(weights(zero, ".shared.down")) > least
    assert moved(weights(lambda v: torch.ones_like(v), ".dq.norm", ".dkv.norm")) > least

    def no_limits(d):
        for layer in d["layers"]:
            if layer["mlp"]:
                layer["mlp"]["expert"]["limit"] = 1e9
    assert moved(cfg2=changed(no_limits)) > least
    assert moved(cfg2=changed(lambda d: [m["mixer"]["rot"].pop("scaling", None) for m in d["layers"]])) > least
    assert moved(cfg2=changed(lambda d: [m["mixer"].update(decay=[1.0] * m["mixer"]["heads"]) for m in d["layers"] if "decay" in m["mixer"]])) > 0.01
    assert moved(cfg2=changed(lambda d: d.update(postln_alpha=1.0))) > 0.01
    rt = load(c, dtype)
    agrees(replay.run_whole(rt, ids), ref, dtype)
    agrees(replay.run_tail(rt, ids, 45), ref, dtype)


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
def test_trace_replay_of_a_teselix_folder(tmp_path, tmp_path_factory):
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
    """The named small configuration (tensor-core products, attention, retention and experts) on a prompt of 2,500
    tokens, then 70 single tokens: too long for the plain implementation, so the engine is held against itself: the
    32-bit logits must not depend on where the prompt ends and the single tokens begin, and bfloat16 must agree with
    32-bit within its rounding."""
    from airframe_b200.config.presets import preset
    folder = make_folder(preset("teselix-small"), seed=4, root=tmp_path_factory.mktemp("txsmall"))
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
