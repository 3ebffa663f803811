"""The kernels behind Teselix's mechanisms, each alone against the plain implementation's functions
(``plain_teselix``, float64): the norm of a residual sum with its gate, copy and shift; the token shift over prompts and
single tokens; the two latents with either pairing of the rotation, stretched frequencies and paged cache rows; retention
token by token, over single tokens in one kernel, and over prompts in chunks on the tensor cores, with one key made to
stand out at chosen distances; and the experts looked up by token, with the shared one beside or among them."""
from types import SimpleNamespace

import pytest
import torch

import plain_teselix as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64
PAGE = 64


@pytest.fixture(scope="module")
def K():
    from airframe_b200 import kernels
    return kernels


def close(got, ref, tol, what=None):
    ref = ref.double().cpu()
    err = float((got.double().cpu() - ref).abs().max() / ref.abs().max().clamp_min(1e-30))
    assert err < tol, (err, what)


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def batch_of(lens, slots, before=None):
    """What the kernels read of a step: sequences packed one after the other, ``before`` tokens seen already."""
    before = before or [0] * len(lens)
    starts, seq, pos = [0], [], []
    for b, n in enumerate(lens):
        starts.append(starts[-1] + n)
        seq += [b] * n
        pos += list(range(before[b], before[b] + n))
    after = [a + n for a, n in zip(before, lens)]
    return SimpleNamespace(seq_starts=i32(starts), slots=i32(slots), n_seqs=len(lens), n_tokens=starts[-1],
                           seq_of_token=i32(seq), positions=i32(pos), len_after=i32(after), is_prefill=not any(before),
                           max_len=max(lens), seq_lens=list(lens), max_len_after=max(after), aux={}, tokens=i32([0] * starts[-1]))


# ---------------------------------------------------------------- the norm of a sum, the shift

@pytest.mark.parametrize("H,T", [(50, 3), (72, 9), (128, 40), (51, 2), (1024, 300), (2052, 5), (5000, 3), (9000, 2), (12000, 2)])
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
def test_norm_of_a_sum(K, H, T, out_dtype):
    g = torch.Generator().manual_seed(H)
    r = lambda *s: torch.randn(*s, generator=g)
    x, w, b, zb, mu = r(T, H) + 2.0, r(H), r(H), r(H), r(H)
    eps, alpha = 1e-5, 1.3
    tol = 2e-5 if out_dtype == torch.float32 else 6e-3
    d = lambda t: t.to(DEV).contiguous()
    y = torch.empty(T, H, dtype=out_dtype, device=DEV)
    K.layer_norm(y, d(x), d(w), d(b), eps)
    close(y, plain.layer_norm(x.double(), w.double(), b.double(), eps), tol)
    rows = [T - 1, 0]
    y2 = torch.empty(2, H, dtype=out_dtype, device=DEV)
    K.layer_norm(y2, d(x), d(w), d(b), eps, rows=i32(rows))
    assert torch.equal(y2, y[rows])
    a16, parts, one, z, zparts = r(T, H).to(torch.bfloat16), r(3, T, H), r(T, H), r(T, H), r(9, T, H)
    slots, n_slots = [(7 * t + 1) % (T + 3) if t != 1 else -1 for t in range(T)], T + 3
    prev = r(n_slots, H)
    for terms, total in (([(d(a16), 1.0)], a16.double()), ([(d(parts), 0.5), (d(one), -2.0)], 0.5 * parts.double().sum(0) - 2.0 * one.double()),
                         ([(d(one), 1.0), (d(parts), 1.0), (d(a16), 3.0)], one.double() + parts.double().sum(0) + 3.0 * a16.double())):
        for gate, zz in ((None, None), (d(z), z.double()), (d(zparts), zparts.double().sum(0))):
            total_g = total if zz is None else total * plain.sigmoid(zz + zb.double())
            ref = plain.norm_of_sum(x.double(), total_g, alpha, w.double(), b.double(), eps)
            for shifted in (False, True):
                xs, st = d(x), d(prev)
                y = torch.empty(T, H, dtype=out_dtype, device=DEV)
                hs = torch.full((T, H), float("nan"), dtype=out_dtype, device=DEV)
                more = dict(shifted=hs, shift=d(mu), prev=st, slots=i32(slots)) if shifted else {}
                K.norm_of_sum(xs, terms, alpha, d(w), d(b), eps, gate=gate, gate_bias=d(zb) if gate is not None else None, y=y, **more)
                close(xs, ref, 2e-5)
                close(y, ref, tol)
                if shifted:
                    before = torch.stack([prev[s].double() if s >= 0 else torch.zeros(H, dtype=F64) for s in slots])
                    close(hs, ref + (before - ref) * mu.double(), tol)
                    want = prev.clone().double()
                    for t, s in enumerate(slots):
                        if s >= 0:
                            want[s] = ref[t]
                    close(st, want, 2e-5)


@pytest.mark.parametrize("H", [128, 50, 2052])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_token_shift_over_prompts_and_single_tokens(K, H, dtype):
    """Two prompts in one step, then single tokens (the state holds the row before), then another sequence in a slot
    used before, whose first token sees zeros; a padding row touches no state."""
    g = torch.Generator().manual_seed(H)
    seqs = {2: torch.randn(9, H, generator=g), 0: torch.randn(1, H, generator=g), 1: torch.randn(4, H, generator=g)}
    mu = torch.rand(H, generator=g)
    ref = {s: plain.shifted(x.double(), mu.double()) for s, x in seqs.items()}
    tol = 1e-6 if dtype == torch.float32 else 6e-3
    state = torch.full((4, H), float("nan"), device=DEV)          # (a slot's state is read only once it has been written)
    fed = {2: 7, 0: 1, 1: 3}

    def run(order, lens, before):
        x = torch.cat([seqs[s][b:b + n] for s, n, b in zip(order, lens, before)]).to(DEV).contiguous()
        h = torch.empty(x.shape[0], H, dtype=dtype, device=DEV)
        y = torch.empty_like(h)
        K.token_shift(h, x, mu.to(DEV), state, batch_of(lens, order, before), y=y)
        close(y, x, tol)
        at = 0
        for s, n, b in zip(order, lens, before):
            close(h[at:at + n], ref[s][b:b + n], tol, (s, b))
            at += n

    run([2, 0, 1], [7, 1, 3], [0, 0, 0])
    for step in range(2):
        order = [2] + ([1] if step == 0 else [])
        run(order, [1] * len(order), [fed[s] + step for s in order])
    close(state[2], seqs[2][8], 1e-6)
    seqs[2] = torch.randn(5, H, generator=g)
    ref[2] = plain.shifted(seqs[2].double(), mu.double())
    run([2], [5], [0])
    kept = state.clone()
    x = torch.randn(1, H, device=DEV)
    h = torch.empty(1, H, dtype=dtype, device=DEV)
    K.token_shift(h, x, mu.to(DEV), state, batch_of([1], [-1], [3]))
    assert torch.equal(state.nan_to_num(7.0), kept.nan_to_num(7.0))


# ---------------------------------------------------------------- the latents

@pytest.mark.parametrize("heads,dim,rot,rank,q_rank,pitch", [(3, 10, 6, 20, 14, 0), (2, 64, 16, 112, 48, 128), (1, 5, 4, 11, 3, 0), (2, 9, 0, 8, 5, 0)])
@pytest.mark.parametrize("pairing", ["half", "adjacent"])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_latents_queries_and_cache_rows(K, heads, dim, rot, rank, q_rank, pitch, pairing, dtype):
    from airframe_b200.config import PartSpec
    from airframe_b200.parts import BuildContext, build_part
    lens = [5, 66]
    T = sum(lens)
    batch = batch_of(lens, [0, 1])
    proj = torch.randn(T, q_rank + rank + rot + 3, device=DEV)
    parts = torch.randn(3, T, heads * (dim + rot), device=DEV)
    norm_w, side_w = torch.randn(rank, device=DEV), torch.randn(q_rank, device=DEV)
    sc = {"factor": 3.0, "original": 30.0, "fast": 8.0, "slow": 0.5}
    rope = build_part("position", PartSpec("rope", {"theta": 77.0, "rotary_dim": rot, "pairing": pairing, "precise_angles": True,
                                                    "scaling": sc}), BuildContext(dtype, torch.device(DEV)))
    rope.load({})
    kc = torch.zeros(4, 1, PAGE, rank + rot, dtype=dtype, device=DEV)
    kv = SimpleNamespace(k=kc, v=None, page_table=i32([[2, -1], [0, 3]]), ring_rows=0)
    P = pitch or dim + rot
    q = torch.full((T, heads * P), float("nan"), dtype=dtype, device=DEV)
    kvrow = torch.empty(T, rank + rot, dtype=dtype, device=DEV)
    side = torch.empty(T, q_rank, dtype=dtype, device=DEV)
    table = rope.precise_table(batch)
    turn = dict(pairing=pairing, magnitude=rope.magnitude, table=table)
    K.latent_prep(batch, heads, dim, rot, rank, 1e-5, rope.inv_freq, side=side, side_src=proj[:, :q_rank], side_w=side_w, kvrow=kvrow,
                  kv_src=proj[:, q_rank: q_rank + rank + rot], norm_w=norm_w, kv=kv, **turn)
    K.latent_prep(batch, heads, dim, rot, rank, 1e-5, rope.inv_freq, q=q, q_src=parts, pitch=pitch, **turn)
    freqs, mag = plain.frequencies({"base": 77.0, "dims": rot, "scaling": sc}) if rot else (torch.zeros(0, dtype=F64), 1.0)
    rotate = plain.rotate_half_split if pairing == "half" else plain.rotate_neighbours
    x, qq = proj.double().cpu(), parts.double().cpu().sum(0).view(T, heads, dim + rot)

    def turned(z):                      # (positions start over with every sequence)
        return torch.cat([rotate(part, freqs, mag) for part in z.split(lens)])

    tol = 3e-6 if dtype == torch.float32 else 8e-3
    close(side, plain.rms(x[:, :q_rank], 1e-5, side_w.double().cpu()), tol)
    c = plain.rms(x[:, q_rank: q_rank + rank], 1e-5, norm_w.double().cpu())
    r = turned(x[:, None, q_rank + rank: q_rank + rank + rot])[:, 0]
    rows = torch.cat([c, r], dim=1)
    close(kvrow, rows, tol)
    ref = torch.zeros(T, heads, P, dtype=F64)
    ref[..., :dim] = qq[..., :dim]
    ref[..., dim: dim + rot] = turned(qq[..., dim:])
    close(q.view(T, heads, P), ref, tol)
    close(kc[2, 0, :5], rows[:5], tol)
    close(kc[0, 0], rows[5:69], tol)
    close(kc[3, 0, :2], rows[69:], tol)
    assert float(kc[1].abs().max()) == 0 and float(kc[3, 0, 2:].abs().max()) == 0
    # without the step's table the angles come from the frequencies in 32 bits: the same rows
    again = torch.empty_like(kvrow)
    K.latent_prep(batch, heads, dim, rot, rank, 1e-5, rope.inv_freq, kvrow=again, kv_src=proj[:, q_rank: q_rank + rank + rot],
                  norm_w=norm_w, pairing=pairing, magnitude=rope.magnitude)
    close(again, rows, max(tol, 2e-5))


# ---------------------------------------------------------------- retention

def _retention_case(heads, dk, dv, n_rot, lens, seed, scaling=None):
    g = torch.Generator().manual_seed(seed)
    T = sum(lens)
    q, k = (torch.randn(T, heads * dk, generator=g) for _ in range(2))
    v, gate = (torch.randn(T, heads * dv, generator=g) for _ in range(2))
    decay = torch.tensor([1.0 - 2.0 ** -(1 + 2 * h) for h in range(heads)], dtype=F64)
    rot = {"base": 40.0, "dims": 2 * n_rot}
    if scaling:
        rot["scaling"] = scaling
    return q, k, v, gate, decay, rot


def _retention_ref(q, k, v, gate, decay, rot, heads, dk, dv, eps, lens):
    """(gated and normed outputs, plain outputs) of every sequence, [T, heads * dv]."""
    freqs, mag = plain.frequencies(rot) if rot["dims"] else (torch.zeros(0, dtype=F64), 1.0)
    ys, os = [], []
    for qs, ks, vs, gs in zip(*(t.double().split(lens) for t in (q, k, v, gate))):
        n = qs.shape[0]
        qr = plain.rotate_half_split(qs.view(n, heads, dk), freqs, mag)
        kr = plain.rotate_half_split(ks.view(n, heads, dk), freqs, mag) * dk ** -0.5
        o = torch.cat([plain.decayed_scan(qr[:, h], kr[:, h], vs.view(n, heads, dv)[:, h], float(decay[h])) for h in range(heads)], 1)
        os.append(o)
        ys.append(torch.cat([plain.rms(p, eps) for p in o.split(dv, dim=1)], 1) * plain.silu(gs))
    return torch.cat(ys), torch.cat(os)


def _table(K, batch, rot):
    if not rot["dims"]:
        return None, 1.0
    freqs, mag = plain.frequencies(rot)
    return K.rope_table_precise(batch.positions, freqs.to(DEV)), mag


SIZES = [(2, 8, 8, 4), (3, 24, 40, 8), (1, 32, 32, 16), (2, 64, 64, 32), (1, 128, 128, 64), (2, 6, 10, 2), (1, 5, 3, 0), (2, 64, 128, 20),
         (1, 128, 64, 64), (1, 256, 96, 128), (1, 192, 192, 96), (2, 40, 33, 3)]


@pytest.mark.parametrize("heads,dk,dv,n_rot", SIZES)
def test_retention_in_every_way(K, heads, dk, dv, n_rot):
    """Four prompts of unequal lengths (one a single token, one that ends one token into a chunk) in one step: token by
    token in 32 bits, and in chunks on the tensor cores, with the norm and gate in the same kernel where it has them;
    then single tokens from the states either of them left, with a padding row, against the plain recurrence."""
    lens, slots, eps, tail = [150, 1, 257, 40], [3, 0, 5, 2], 1e-5, 6
    full = [n + tail for n in lens]
    scaling = {"factor": 4.0, "original": 32.0, "fast": 8.0, "slow": 1.0} if dk == 64 else None
    q, k, v, gate, decay, rot = _retention_case(heads, dk, dv, n_rot, full, dk * 7 + dv, scaling)
    y_ref, o_ref = _retention_ref(q, k, v, gate, decay, rot, heads, dk, dv, eps, full)
    starts = [sum(full[:i]) for i in range(len(full))]
    prompt_rows = torch.cat([torch.arange(s, s + n) for s, n in zip(starts, lens)])
    d = lambda t, rows: t[rows].to(DEV).contiguous()
    f32 = torch.float32
    dec = decay.to(f32).to(DEV)
    scale = dk ** -0.5
    pads = heads * (2 * dk + 2 * dv) + 4
    packed = torch.zeros(prompt_rows.numel(), pads + (-pads) % 4, device=DEV)      # (sections of one projection row)
    n_k, n_v = heads * dk, heads * dv
    off = [0, n_k, 2 * n_k, 2 * n_k + n_v]
    for o, t in zip(off, (q, k, v, gate)):
        packed[:, o: o + t.shape[1]] = d(t, prompt_rows)
    qs, ks, vs, gs = (packed[:, o: o + n] for o, n in zip(off, (n_k, n_k, n_v, n_v)))
    results = {}
    for way in ("scan", "chunks"):
        state = torch.zeros(6, heads, dv, dk, device=DEV)
        state[1] = 7.0                                                # (nobody's slot)
        batch = batch_of(lens, slots)
        table, mag = _table(K, batch, rot)
        T = batch.n_tokens
        if way == "scan":
            qc, kc = qs.clone(), ks.clone()
            if table is not None:
                K.rotate_rows(qc, kc, table, heads, dk, magnitude=mag)
            o = torch.empty(T, n_v, device=DEV)
            K.state_scan("decay", o, qc, kc, vs, state, batch, heads, dk, dv, decay=dec)
            close(o * scale, o_ref[prompt_rows], 2e-5, way)
            y = torch.empty(T, n_v, device=DEV)
            K.gated_group_norm(y, o, None, gs, dv, eps, gate_act="silu", in_scale=scale)
            close(y, y_ref[prompt_rows], 5e-5, way)
        else:
            powers = (decay[:, None] ** torch.arange(K.RETENTION_CHUNK + 1, dtype=F64)).to(f32).to(DEV).contiguous()
            o = torch.empty(T, n_v, device=DEV)
            K.retention_prompt(o, qs, ks, vs, None, table, powers, state, batch, heads, dk, dv, scale, eps, magnitude=mag)
            close(o, o_ref[prompt_rows], 1e-4, way)
            if dv <= 128:
                kept = state.clone()
                state.zero_()
                y = torch.empty(T, n_v, dtype=torch.bfloat16, device=DEV)
                K.retention_prompt(y, qs, ks, vs, gs, table, powers, state, batch, heads, dk, dv, scale, eps, magnitude=mag)
                close(y, y_ref[prompt_rows], 8e-3, way)
                assert torch.equal(state[slots], kept[slots])         # (the same sums)
                state[1] = 7.0
        assert float((state[1] - 7.0).abs().max()) == 0
        results[way] = state
    close(results["chunks"][slots], results["scan"][slots].double(), 1e-4)
    # single tokens, from the states the token-by-token scan left; one padding row in between
    for out_dtype in (f32, torch.bfloat16):
        state = results["scan"].clone()
        for i in range(tail):
            rows = torch.tensor([starts[0] + lens[0] + i, starts[1] + lens[1] + i, 0, starts[2] + lens[2] + i, starts[3] + lens[3] + i])
            batch = batch_of([1] * 5, [slots[0], slots[1], -1, slots[2], slots[3]], [lens[0] + i, lens[1] + i, 0, lens[2] + i, lens[3] + i])
            table, mag = _table(K, batch, rot)
            y = torch.full((5, n_v), float("nan"), dtype=out_dtype, device=DEV)
            K.retention_step(y, d(q, rows), d(k, rows), d(v, rows), d(gate, rows), table, dec, state, batch, heads, dk, dv, scale, eps,
                             magnitude=mag)
            live = [0, 1, 3, 4]
            close(y[live], y_ref[rows[live]], 5e-5 if out_dtype == f32 else 8e-3, i)
            assert float(y[2].abs().max()) == 0
        assert float((state[1] - 7.0).abs().max()) == 0


@pytest.mark.parametrize("far", [1, 63, 64, 65, 127, 128, 129, 300])
def test_retention_sees_a_loud_key_at_every_distance(K, far):
    """One key and the query ``far`` tokens on stand out (equal, scaled up, everything else small): the output there is
    that key's value times the decay to that power, the query right before the key does not see it, and a chunk's or a
    tile's border between them changes nothing.  On the tensor cores against the plain recurrence."""
    heads, dk, dv, T = 1, 64, 64, 420
    g = torch.Generator().manual_seed(far)
    q, k, v = torch.randn(T, dk, generator=g) * 0.002, torch.randn(T, dk, generator=g) * 0.002, torch.randn(T, dv, generator=g)
    at = 70
    loud = torch.randn(dk, generator=g) * 5.0
    k[at] = loud
    q[at + far] = loud
    q[at - 1] = loud
    decay = torch.tensor([0.99], dtype=F64)
    o_ref = plain.decayed_scan(q.double(), k.double(), v.double(), 0.99)
    powers = (decay[:, None] ** torch.arange(K.RETENTION_CHUNK + 1, dtype=F64)).float().to(DEV).contiguous()
    state = torch.zeros(1, 1, dv, dk, device=DEV)
    o = torch.empty(T, dv, device=DEV)
    K.retention_prompt(o, q.to(DEV), k.to(DEV), v.to(DEV), None, None, powers, state, batch_of([T], [0]), heads, dk, dv, 1.0, 1e-5)
    expect = float(loud.double() @ loud.double()) * 0.99 ** far * v[at].double()
    close(o_ref[at + far], expect, 2e-2)
    close(o[at + far], o_ref[at + far], 1e-4)
    close(o[at - 1], o_ref[at - 1], 1e-4)
    assert float(o_ref[at - 1].abs().max()) < 0.2 * float(o_ref[at + far].abs().max())
    S = torch.zeros(dk, dv, dtype=F64)
    for t in range(T):
        S = 0.99 * S + k[t].double()[:, None] * v[t].double()[None]
    close(state[0, 0], S.T, 1e-4)


# ---------------------------------------------------------------- experts looked up by token

@pytest.mark.parametrize("E,top,f,sf,width,T", [(5, 2, 36, 40, 72, 7), (4, 1, 64, 64, 128, 9), (8, 3, 64, 128, 128, 300), (3, 3, 22, 10, 50, 40),
                                                (1, 1, 17, None, 51, 5), (16, 2, 64, 60, 64, 1), (6, 2, 32, 96, 64, 70)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_experts_looked_up_by_token(K, E, top, f, sf, width, T, dtype):
    from airframe_b200.config import PartSpec
    from airframe_b200.parts import BuildContext, build_part
    from airframe_b200.parts.linear import as_terms
    g = torch.Generator().manual_seed(E * 100 + f)
    V = 23
    params = {"hidden_size": width, "intermediate_size": f, "num_experts": E, "top": top, "limit": 0.9, "table_weight": "table",
              "vocab_size": V, "expert_weights": "e{e}.{role}"}
    if sf is not None:
        params["shared"] = {"intermediate_size": sf, "limit": 0.4, "gate_weight": "shared.gate", "up_weight": "shared.up",
                            "down_weight": "shared.down"}
    parts = [build_part("feed_forward", PartSpec("routed_experts", params), BuildContext(dtype, torch.device(DEV))) for _ in range(2)]
    W = []
    for part in parts:
        w = {}
        for decl in part.weight_decls():
            if decl.name == "table":
                w["table"] = torch.rand(V, E, generator=g).argsort(dim=1)[:, :top].to(torch.int32)
            else:
                w[decl.name] = (torch.randn(*decl.shape, generator=g) * (1.5 / decl.shape[1] ** 0.5)).to(torch.bfloat16).float()
        part.load({n: t.to(DEV) for n, t in w.items()})
        W.append({n: (t.double() if n != "table" else t) for n, t in w.items()})
    assert parts[0].joined == {36: 0, 64: -(-(sf or 0) // 64), 22: 0, 17: 0, 32: 3}[f]
    type(parts[0]).link(parts)
    tokens = torch.randint(0, V, (T,), generator=g)
    x = torch.randn(T, width, generator=g).to(torch.bfloat16).float()
    batch = batch_of([T], [0])
    batch.tokens = tokens.to(torch.int32).to(DEV)
    mlp = {"router": {"top": top}, "expert": {"limit": 0.9}}
    if sf is not None:
        mlp["shared"] = {"limit": 0.4}
    for part, w in zip(parts, W):                       # (both layers' plans come out of one kernel, at the first of them)
        got = sum(s * (t.double().sum(0) if t.dim() == 3 else t.double()) for t, s in as_terms(part.forward(x.to(DEV).to(dtype), batch)))
        close(got, plain.table_experts(x.double(), tokens.tolist(), w, "", mlp), 1e-5 if dtype == torch.float32 else 8e-3)
    assert len([k for k in batch.aux if k[0] == "expert_plans"]) == 1


def test_a_table_must_name_experts_that_exist(K):
    from airframe_b200.config import ConfigError, PartSpec
    from airframe_b200.parts import BuildContext, build_part
    params = {"hidden_size": 8, "intermediate_size": 8, "num_experts": 2, "top": 1, "limit": 1.0, "table_weight": "table",
              "vocab_size": 3, "expert_weights": "e{e}.{role}"}
    part = build_part("feed_forward", PartSpec("routed_experts", params), BuildContext(torch.float32, torch.device(DEV)))
    w = {d.name: torch.zeros(*d.shape, device=DEV) for d in part.weight_decls()}
    w["table"] = i32([[0], [1], [2]])
    with pytest.raises(ConfigError):
        part.load(w)
