"""The kernels behind Retudra's mechanisms, each alone against the plain implementation's functions (``plain_retudra``,
float64): attention with a window that keeps first tokens, over prompts and over paged rings, with one key made to stand out
at the edges; the convolution, the decays and the delta rule over prompts and single tokens; the router with softmax scores,
groups by their largest and identity experts; experts with a SiLU gate; the norm on a sublayer's output; a token's own gated
row; a gate per value."""
import math
from types import SimpleNamespace

import pytest
import torch

import plain_retudra as plain

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


# ---------------------------------------------------------------- windows that keep first tokens

WINDOWS = [(1, 1), (10, 3), (64, 64), (65, 63), (100, 70), (128, 65), (130, 128), (300, 5)]


@pytest.mark.parametrize("size,keep", WINDOWS)
@pytest.mark.parametrize("hd,nq,nkv,dtype", [(24, 3, 1, torch.float32), (48, 4, 2, torch.bfloat16), (64, 4, 2, torch.bfloat16),
                                             (128, 4, 1, torch.bfloat16), (256, 2, 2, torch.bfloat16)])
def test_prompts_under_a_window_with_kept_tokens(K, size, keep, hd, nq, nkv, dtype):
    """Unequal prompts in one step; at every edge (the last kept position, the one behind it, the window's first, the one
    before it) a key that would win its query's softmax alone."""
    lens = [330, 1, 70, 200]
    T = sum(lens)
    g = torch.Generator().manual_seed(size * 3 + keep + hd)
    q, k, v = (torch.randn(T, n, hd, generator=g) for n in (nq, nkv, nkv))
    scale = 1.0 / math.sqrt(hd)
    edges = [keep - 1, keep, 330 - 1 - size + 1, 330 - 1 - size]            # seen from position 329 of the first prompt
    batch = batch_of(lens, [0, 1, 2, 3])
    for e in edges:
        if not 0 <= e < 330:
            continue
        kk = k.clone()
        kk[e, 0] = q[329, 0] * (12.0 * math.sqrt(hd) / float(q[329, 0].pow(2).sum()))        # a score of 12 above the rest
        qd, kd, vd = (t.to(dtype).to(DEV).reshape(T, -1).contiguous() for t in (q, kk, v))
        out = torch.full((T, nq * hd), float("nan"), dtype=dtype, device=DEV)
        K.attn_prefill(out, qd, kd, vd, batch, nq, nkv, hd, scale, 0.0, size, keep=keep)
        K.check_device_errors(DEV)
        row = 0
        for n in lens:
            r = slice(row, row + n)
            ref = plain.attend(*(t.to(dtype).double()[r] for t in (q, kk, v)), scale, plain.visible(n, size, keep))
            assert float((out[r].double().cpu() - ref).abs().max()) < (1e-5 if dtype == torch.float32 else 2e-2), (e, n)
            row += n


@pytest.mark.parametrize("size,keep", WINDOWS)
@pytest.mark.parametrize("hd,nq,nkv,dtype", [(24, 3, 1, torch.float32), (48, 4, 2, torch.bfloat16), (64, 6, 2, torch.bfloat16),
                                             (128, 20, 1, torch.bfloat16), (256, 2, 2, torch.bfloat16)])
@pytest.mark.parametrize("plan", [False, True])
def test_decoding_over_a_ring_behind_kept_pages(K, size, keep, hd, nq, nkv, dtype, plan):
    """Rows stored by the cache kernel (a prompt longer than pages and ring together, then single tokens), pages scrambled;
    a padding row; a key that stands out at every edge, where the window sees it and where it does not."""
    from airframe_b200.cache.sequence_cache import KVView
    from airframe_b200.parts.base import KVNeed
    g = torch.Generator().manual_seed(size + keep * 5 + hd)
    ring, kept = -(-size // PAGE) * PAGE, -(-keep // PAGE) * PAGE
    per = (ring + kept) // PAGE
    lens = [500, 3, 129, 64, 257]
    B = len(lens)
    scale = 1.0 / math.sqrt(hd)
    q = torch.randn(B, nq, hd, generator=g)
    ks, vs = [torch.randn(n, nkv, hd, generator=g) for n in lens], [torch.randn(n, nkv, hd, generator=g) for n in lens]
    order = torch.randperm(B * per, generator=g).view(B, per) + 1
    for e in {keep - 1, keep, 500 - size, 500 - size - 1, 499} & set(range(500)):
        ks[0] = ks[0].clone()
        old = ks[0][e].clone()
        ks[0][e, 0] = q[0, 0] * (12.0 * math.sqrt(hd) / float(q[0, 0].pow(2).sum()))
        kc = torch.full((B * per + 1, nkv, PAGE, hd), 7.0, dtype=dtype, device=DEV)
        vc = torch.full_like(kc, 7.0)
        kv = KVView(kc, vc, i32(order.tolist()), ring, KVNeed(nkv, hd, size, keep_first=keep), keep)
        # all but the last token in one step, the last one by itself
        for first in (True, False):
            cut = [(n - 1 if first else 1) for n in lens]
            bt = batch_of([c for c in cut if c], [i for i, c in enumerate(cut) if c], None if first else [n - 1 for n in lens])
            rows = torch.cat([torch.cat([torch.zeros(c, nq * hd), (k[:-1] if first else k[-1:]).reshape(c, -1),
                                         (v[:-1] if first else v[-1:]).reshape(c, -1)], 1) for c, k, v in zip(cut, ks, vs) if c])
            K.store_kv(rows.to(dtype).to(DEV), bt, nq, nkv, hd, kv)
        batch = SimpleNamespace(slots=i32([*range(B), -1]), len_after=i32([*lens, 0]), max_len_after=500, n_seqs=B + 1)
        if plan:
            batch.aux = {}
        out = torch.full((B + 1, nq * hd), float("nan"), dtype=dtype, device=DEV)
        qd = torch.cat([q.reshape(B, -1), torch.zeros(1, nq * hd)]).to(dtype).to(DEV)
        K.attn_decode(out, qd, kv, batch, nq, nkv, hd, scale, 0.0, size)
        K.check_device_errors(DEV)
        for b, n in enumerate(lens):
            full = torch.zeros(n, nq, hd, dtype=F64)
            full[-1] = q[b].to(dtype).double()
            ref = plain.attend(full, ks[b].to(dtype).double(), vs[b].to(dtype).double(), scale, plain.visible(n, size, keep))[-1]
            assert float((out[b].double().cpu() - ref).abs().max()) < (1e-5 if dtype == torch.float32 else 2e-2), (e, b)
        assert float(out[B].float().abs().max()) == 0.0
        ks[0][e] = old


# ---------------------------------------------------------------- the delta rule behind a decay per key channel

def _delta_case(lens, G, H, dk, dv, taps, seed, aligned):
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    C = 2 * G * dk + H * dv
    T = sum(lens)
    offs, at = [], 4 if aligned else 2
    for n in (G * dk, G * dk, H * dv, H):                  # sections with gaps, on 16 bytes or not
        offs.append(at)
        at += n + 3
        if aligned:
            at = -(-at // 4) * 4
    return SimpleNamespace(proj=r(T, at), offs=offs, taps=r(C, taps), C=C, T=T, r=r)


def _ref_conv(c, rows, G, H, dk, dv, taps):
    """[q | k | v | beta] of one whole sequence (its projection rows)."""
    nq = G * dk
    secs = [rows[:, o: o + n] for o, n in zip(c.offs, (nq, nq, H * dv, H))]
    x = plain.silu(plain.short_conv(torch.cat(secs[:3], 1).double(), c.taps.double()))
    n = rows.shape[0]
    q = plain.unit(x[:, :nq].view(n, G, dk)) * 0.3
    k = plain.unit(x[:, nq: 2 * nq].view(n, G, dk))
    return torch.cat([q.reshape(n, nq), k.reshape(n, nq), x[:, 2 * nq:], plain.sigmoid(secs[3].double())], 1)


@pytest.mark.parametrize("G,H,dk,dv,taps", [(2, 4, 12, 20, 3), (1, 3, 64, 64, 4), (1, 1, 5, 3, 9), (3, 3, 128, 128, 2), (2, 2, 192, 96, 4),
                                            (1, 2, 300, 10, 1), (2, 2, 32, 48, 1), (1, 1, 520, 8, 5), (3, 6, 16, 10, 3),
                                            (5, 5, 4, 4, 4), (18, 18, 128, 128, 4), (1, 1, 8, 20, 2)])
@pytest.mark.parametrize("aligned", [False, True])
def test_convolution_unit_keys_and_step_sizes(K, G, H, dk, dv, taps, aligned):
    """Prompts of unequal lengths (one and two tokens among them: shorter than the convolution reaches), then single tokens one
    by one with the history carried on, a slot used again, a padding row."""
    lens, tail = [40, 1, 2, 17], 12
    full = [n + tail for n in lens]
    c = _delta_case(full, G, H, dk, dv, taps, dk + taps, aligned)
    wide = lambda T: torch.empty(T, -(-(c.C + H) // 4) * 4, device=DEV)[:, : c.C + H]
    seqs, at = [], 0
    for n in full:
        seqs.append(c.proj[at: at + n])
        at += n
    refs = [_ref_conv(c, s, G, H, dk, dv, taps) for s in seqs]
    tw = c.taps.t().contiguous().to(DEV)
    slots = [3, 0, 2, 5]
    for again in range(2):
        hist = torch.zeros(6, max(taps - 1, 1), c.C, device=DEV) if not again else hist
        if again:
            hist.zero_()                                    # (what taking a slot does)
        out = wide(sum(lens))
        low = torch.empty(sum(lens), 24, dtype=torch.bfloat16, device=DEV)
        rows = torch.cat([s[:n] for s, n in zip(seqs, lens)])
        K.delta_conv(out, rows.to(DEV), c.offs, tw, hist if taps > 1 else None, batch_of(lens, slots), G, H, dk, dv, 1e-6, 0.3,
                     low=low, low_sections=((0, 5, 0), (2, 7, 8)))
        assert torch.equal(low[:, :5].cpu(), rows[:, :5].bfloat16()) and torch.equal(low[:, 8:15].cpu(), rows[:, 2:9].bfloat16())
        close(out, torch.cat([r[:n] for r, n in zip(refs, lens)]), 2e-5)
        for j in range(tail):
            b = batch_of([1] * 5, [*slots, -1], [*(n + j for n in lens), 0])
            step = torch.cat([*(s[n + j: n + j + 1] for s, n in zip(seqs, lens)), torch.ones(1, c.proj.shape[1])]).to(DEV)
            out = wide(5)
            K.delta_conv(out, step, c.offs, tw, hist if taps > 1 else None, b, G, H, dk, dv, 1e-6, 0.3)
            close(out[:4], torch.cat([r[n + j: n + j + 1] for r, n in zip(refs, lens)]), 2e-5, j)
        if taps > 1:
            assert float(hist[[1, 4]].abs().max()) == 0.0   # nobody else's history


@pytest.mark.parametrize("T,rank,n", [(3, 10, 48), (40, 24, 130), (16, 7, 33), (300, 96, 256)])
def test_decays_of_every_kind(K, T, rank, n):
    g = torch.Generator().manual_seed(T)
    r = lambda *s: torch.randn(*s, generator=g)
    proj, w2, bias, rate = r(T, rank + 9), r(n, rank), r(n) * 10.0, torch.rand(n, generator=g) * 5.0
    z = proj[:, 4: 4 + rank].double() @ w2.double().T
    d = lambda t: t.to(DEV).contiguous()
    out = torch.empty(T, n, device=DEV)
    K.channel_decay(out, d(proj), 4, d(w2.t()), d(bias), kind="softplus", rate=d(rate))
    close(out, torch.exp(-rate.double() * plain.softplus(z + bias.double())), 2e-5)
    K.channel_decay(out, d(proj), 4, d(w2.t()), None, kind="logit")
    close(out, z, 1e-5)
    K.channel_decay(out, d(proj), 4, d(w2.t()), d(bias), tau=3.0)
    close(out, plain.sigmoid(z + bias.double()) ** (1.0 / 3.0), 2e-5)
    with pytest.raises(K.KernelError):
        K.channel_decay(out, d(proj), 4, d(w2.t()), d(bias), kind="softplus")
    if T <= K.DECAY_FEW:                                      # both in one kernel, ranks and sizes apart
        g2, gate = r(n + 45, rank + 3), torch.empty(T, n + 45, device=DEV)
        K.decay_and_gate(out, gate, d(proj), 4, d(w2.t()), d(bias), d(rate), 5, d(g2.t()))
        close(out, torch.exp(-rate.double() * plain.softplus(z + bias.double())), 2e-5)
        close(gate, proj[:, 5: 8 + rank].double() @ g2.double().T, 1e-5)


def delta_inputs(T, G, H, dk, dv, seed, keep=None):
    """Unit queries and keys, values, decays from 0 to 1 (``keep``: all of them that), step sizes."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    q, k = plain.unit(r(T, G, dk).double()).float(), plain.unit(r(T, G, dk).double()).float()
    w = torch.exp(-torch.exp(2.0 * r(H, dk)) * torch.rand(T, H, dk, generator=g)) if keep is None else torch.full((T, H, dk), keep)
    w[:, 0, :1] = 0.0                                         # a channel that keeps nothing
    w[:, 0, dk - 1:] = 1.0                                    # and one that keeps everything
    return q, k, r(T, H, dv), w, torch.rand(T, H, generator=g)


def ref_scan(q, k, v, w, beta):
    H, G = v.shape[1], q.shape[1]
    o = [plain.delta_scan(*(t.double() for t in (q[:, h // (H // G)], k[:, h // (H // G)], v[:, h], w[:, h], beta[:, h])))
         for h in range(H)]
    return torch.stack(o, 1)


DELTA_SHAPES = [(2, 4, 12, 20), (1, 1, 5, 3), (1, 3, 64, 64), (2, 2, 128, 128), (1, 2, 192, 96), (3, 3, 10, 6), (1, 2, 32, 200), (1, 1, 256, 64)]


@pytest.mark.parametrize("G,H,dk,dv", DELTA_SHAPES)
def test_delta_rule_token_by_token(K, G, H, dk, dv):
    """Unequal prompts in one step, then single tokens from the states they left, with a padding row."""
    lens, tail = [37, 1, 90], 5
    full = [n + tail for n in lens]
    parts = [delta_inputs(n, G, H, dk, dv, 9 * n + dk) for n in full]
    refs = [ref_scan(*p) for p in parts]
    state = torch.zeros(4, H, dv, dk, device=DEV)

    def run(pick, batch, pad=0):
        rows = [torch.cat([p[i][s].flatten(1) for p, s in zip(parts, pick)] + ([torch.zeros(pad, parts[0][i][0].numel())] if pad else []))
                for i in range(5)]
        q, k, v, w, beta = (t.to(DEV).contiguous() for t in rows)
        out = torch.full((q.shape[0], H * dv), float("nan"), device=DEV)
        K.state_scan("gated", out, q, k, v, state, batch, H, dk, dv, w=w, beta=beta)
        return out

    out = run([slice(0, n) for n in lens], batch_of(lens, [2, 0, 3]))
    close(out, torch.cat([r[:n].flatten(1) for r, n in zip(refs, lens)]), 2e-5)
    for j in range(tail):
        out = run([slice(n + j, n + j + 1) for n in lens], batch_of([1] * 4, [2, 0, 3, -1], [*(n + j for n in lens), 0]), pad=1)
        close(out[:3], torch.cat([r[n + j: n + j + 1].flatten(1) for r, n in zip(refs, lens)]), 2e-5, j)
        assert float(out[3].abs().max()) == 0.0
    assert float(state[1].abs().max()) == 0.0


def _chunked_run(K, parts, picks, batch, state, H, dk, dv, G, tile=0):
    """:func:`kernels.delta_prompt` on rows whose logits give the parts' decays (rate 1, softplus inverted)."""
    rows = [torch.cat([p[i][s].flatten(1) for p, s in zip(parts, picks)]) for i in range(5)]
    q, k, v, w, beta = rows
    lg = -torch.log(w.double().clamp_min(1e-30))                          # softplus(z + bias) is to be this
    z = torch.where(lg > 30.0, lg, torch.log(torch.expm1(lg.clamp(1e-9, 60.0)))).float()
    bias = torch.linspace(-1.0, 1.0, H * dk)
    mixed = torch.cat([q, k, v, beta, torch.zeros(q.shape[0], (-(q.shape[1] * 2 + v.shape[1] + H)) % 4)], 1).to(DEV)
    n = q.shape[1]
    out = torch.full((q.shape[0], H * dv), float("nan"), device=DEV)
    K.delta_prompt(out, mixed[:, :n], mixed[:, n: 2 * n], mixed[:, 2 * n: 2 * n + H * dv], mixed[:, 2 * n + H * dv: 2 * n + H * dv + H],
                   (z - bias).to(DEV).contiguous(), bias.to(DEV), torch.ones(H * dk, device=DEV), state, batch, H, dk, dv, tile=tile)
    K.check_device_errors(DEV)
    return out


CHUNK_SHAPES = [(1, 3, 64, 64), (2, 2, 128, 128), (1, 2, 192, 96), (1, 2, 32, 208), (1, 1, 256, 64), (3, 3, 16, 16), (1, 4, 112, 48), (2, 2, 240, 80)]


@pytest.mark.parametrize("G,H,dk,dv", CHUNK_SHAPES)
@pytest.mark.parametrize("keep,tile", [(None, 16), (None, 32), (1.0, 32), (0.99, 0)])
def test_delta_rule_in_chunks(K, G, H, dk, dv, keep, tile):
    """Prompts of one token, of a group and a token, of a chunk and a token, of whole chunks and of many; decays from nothing to
    everything, none at all, and slow ones; then single tokens from the states the chunks left; slots in any order."""
    assert K.delta_prompt_supported(dk, dv) and not K.delta_prompt_supported(dk + 1, dv) and not K.delta_prompt_supported(dk, dv + 8)
    lens, tail = [1, 17, 33, 64, 230, 16, 31], 3
    full = [n + tail for n in lens]
    parts = [delta_inputs(n, G, H, dk, dv, 5 * n + dk, keep) for n in full]
    refs = [ref_scan(*p) for p in parts]
    slots = [6, 2, 0, 5, 1, 7, 3]
    state = torch.zeros(8, H, dv, dk, device=DEV)
    out = _chunked_run(K, parts, [slice(0, n) for n in lens], batch_of(lens, slots), state, H, dk, dv, G, tile)
    row = 0
    for n, r in zip(lens, refs):
        close(out[row: row + n], r[:n].flatten(1), 2e-4, n)
        row += n
    assert float(state[4].abs().max()) == 0.0
    for j in range(tail):
        rows = [torch.cat([p[i][n + j: n + j + 1].flatten(1) for p, n in zip(parts, lens)]).to(DEV).contiguous() for i in range(5)]
        step = torch.empty(len(lens), H * dv, device=DEV)
        K.state_scan("gated", step, rows[0], rows[1], rows[2], state, batch_of([1] * len(lens), slots, [n + j for n in lens]), H, dk, dv,
                     w=rows[3], beta=rows[4])
        close(step, torch.cat([r[n + j: n + j + 1].flatten(1) for r, n in zip(refs, lens)]), 2e-4, j)


def test_a_prompt_in_two_steps_of_chunks(K):
    """The second step goes on from the states the first one left (both in chunks that end inside a group)."""
    G, H, dk, dv = 1, 2, 64, 64
    p = delta_inputs(150, G, H, dk, dv, 3)
    ref = ref_scan(*p).flatten(1)
    state = torch.zeros(3, H, dv, dk, device=DEV)
    a = _chunked_run(K, [p], [slice(0, 83)], batch_of([83], [1]), state, H, dk, dv, G)
    b = _chunked_run(K, [p], [slice(83, 150)], batch_of([67], [1]), state, H, dk, dv, G)
    close(torch.cat([a, b]), ref, 2e-4)


@pytest.mark.parametrize("back", [1, 5, 15, 16, 17, 31, 32, 33, 48, 64, 200])
def test_one_key_stands_out_in_chunks(K, back):
    """A query asks for one earlier key (orthogonal to all others) ``back`` tokens on: its value comes out, decayed by every
    channel's product in between, and the query right before the key sees nothing of it."""
    G, H, dk, dv, T = 1, 1, 64, 32, 260
    g = torch.Generator().manual_seed(back)
    at = 230 - back
    k = torch.zeros(T, G, dk)
    k[:, :, :32] = torch.randn(T, G, 32, generator=g)
    q = plain.unit(k.double()).float()
    k = q.clone()
    k[at] = 0.0
    k[at, 0, 40:44] = 0.5                                    # a unit key in channels that nobody else uses
    q[230, 0], q[at - 1, 0] = k[at, 0], k[at, 0]
    v = torch.randn(T, H, dv, generator=g)
    w = torch.full((T, H, dk), 0.995)
    w[:, 0, 41] = 0.98
    beta = torch.rand(T, H, generator=g)
    beta[at] = 1.0
    state = torch.zeros(1, H, dv, dk, device=DEV)
    out = _chunked_run(K, [(q, k, v, w, beta)], [slice(0, T)], batch_of([T], [0]), state, H, dk, dv, G).cpu().double()
    want = v[at, 0].double() * (3 * 0.25 * 0.995 ** back + 0.25 * 0.98 ** back)
    assert float((out[230] - want).abs().max()) < 2e-4 and float(out[at - 1].abs().max()) < 1e-5
    close(out, ref_scan(q, k, v, w, beta).flatten(1), 2e-4)


# ---------------------------------------------------------------- experts

@pytest.mark.parametrize("E,ident,top,groups,keep", [(7, 2, 3, 3, 2), (6, 2, 4, 2, 1), (3, 5, 4, 2, 2), (5, 0, 5, 1, 1), (1, 4, 2, 1, 1), (40, 8, 6, 8, 3)])
@pytest.mark.parametrize("T,H,dtype", [(5, 51, torch.float32), (300, 96, torch.bfloat16)])
def test_router_with_softmax_scores(K, E, ident, top, groups, keep, T, H, dtype):
    """Choices and weights, with corrections that make choice scores negative in whole groups."""
    g = torch.Generator().manual_seed(E + top)
    n = E + ident
    h = torch.randn(T, H, generator=g).to(dtype)
    router = torch.randn(n, H, generator=g)
    for shift in (0.0, -1.0):
        corr = torch.randn(n, generator=g) * 0.2 + shift
        ids = torch.empty(T, top, dtype=torch.int32, device=DEV)
        wts = torch.empty(T, top, device=DEV)
        K.expert_route(ids, wts, None, h.to(DEV), router.to(DEV), n, correction=corr.to(DEV), groups=groups, keep=keep,
                       score="softmax", group_score="max")
        s = torch.softmax(h.double() @ router.double().T, -1)
        for t in range(T):
            want = plain.choose(s[t], corr.double(), top, groups, keep)
            assert ids[t].tolist() == want, t
            assert float((wts[t].cpu().double() - s[t, want]).abs().max()) < 1e-5
        if not K.route_plans_fit(T, n, groups):
            continue
        # the same choices with the plan in the same kernel: every pair once, by expert, the identity experts' last
        perm = torch.full((T * top,), -1, dtype=torch.int32, device=DEV)
        plan = torch.empty(1 + 3 * K.expert_max_tiles(T * top, E, 16), dtype=torch.int32, device=DEV)
        ids2, wts2 = torch.empty_like(ids), torch.empty_like(wts)
        K.expert_route(ids2, wts2, None, h.to(DEV), router.to(DEV), n, correction=corr.to(DEV), groups=groups, keep=keep,
                       score="softmax", group_score="max", plan_out=(perm, plan, E, 16))
        assert torch.equal(ids2, ids) and torch.equal(wts2, wts)
        order = perm.cpu().long()
        assert sorted(order.tolist()) == list(range(T * top))
        by = ids.cpu().flatten()[order].clamp(max=E)
        assert torch.equal(by, by.sort().values)
        cells = plan.cpu().tolist()
        covered = []
        for i in range(cells[0]):
            e, r0, m = cells[1 + 3 * i: 4 + 3 * i]
            assert 0 < m <= 16 and by[r0: r0 + m].tolist() == [e] * m
            covered += range(r0, r0 + m)
        assert covered == list(range(int((by < E).sum())))
    with pytest.raises(K.KernelError):
        K.expert_route(ids, wts, None, h.to(DEV), router.to(DEV), n, score="cosine")


@pytest.mark.parametrize("H,F,E,ident,top,T", [(72, 28, 7, 2, 3, 40), (64, 64, 6, 2, 4, 300), (50, 22, 2, 1, 3, 9), (128, 96, 8, 2, 2, 8),
                                               (51, 17, 1, 4, 2, 5), (192, 48, 4, 2, 2, 700)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_experts_with_silu_gates_beside_identity_experts(K, H, F, E, ident, top, T, dtype):
    from airframe_b200.config.base import PartSpec
    from airframe_b200.parts import BuildContext, build_part
    g = torch.Generator().manual_seed(H + T)
    r = lambda *s: torch.randn(*s, generator=g)
    params = {"hidden_size": H, "intermediate_size": F, "num_experts": E, "top": top, "expert": "silu_glu", "router_weight": "router",
              "expert_weights": "e{e}.{role}", "router": {"score": "softmax", "correction_weight": "correction", "identity": ident}}
    W = {"router": r(E + ident, H), "correction": r(E + ident) * 0.1}
    for e in range(E):
        W.update({f"e{e}.gate": r(F, H) * 0.2, f"e{e}.up": r(F, H) * 0.2, f"e{e}.down": r(H, F) * 0.2})
    W = {n: t.to(torch.bfloat16).float() for n, t in W.items()}
    ctx = BuildContext(compute_dtype=dtype, device=torch.device(DEV))
    part = build_part("feed_forward", PartSpec("routed_experts", params), ctx)
    part.load({n: t.to(DEV) for n, t in W.items()})
    h = r(T, H).to(dtype)
    from airframe_b200.parts.linear import as_terms
    out = torch.zeros(T, H, device=DEV)
    K.add_scaled_rmsnorm(out, as_terms(part.forward(h.to(DEV), batch_of([T], [0]))))
    K.check_device_errors(DEV)
    ref = plain.experts(h.double(), {n: t.double() for n, t in W.items()}, "", {"router": {"experts": E, "identity": ident, "top": top}})
    close(out, ref, 2e-5 if dtype == torch.float32 else 1.5e-2)
    assert part.decode_bytes([1]) > 0 and part.prefill_flops([T]) > 0


# ---------------------------------------------------------------- norms and gates

@pytest.mark.parametrize("H,T", [(50, 3), (72, 9), (128, 40), (51, 2), (1024, 300), (2052, 5), (5000, 3), (9000, 2), (12000, 2)])
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
def test_norm_on_a_sublayers_output(K, H, T, out_dtype):
    """x += norm(terms): one tensor, partial sums, two and three scaled terms; the copy of the new row."""
    g = torch.Generator().manual_seed(H)
    r = lambda *s: torch.randn(*s, generator=g)
    x, w, b = r(T, H) + 2.0, r(H), r(H)
    cases = [[(r(T, H), 1.0)], [(r(T, H).to(torch.bfloat16), 1.0)], [(r(5, T, H), 1.0)], [(r(3, T, H), 0.5), (r(T, H), 2.0)],
             [(r(T, H), 0.5), (r(T, H), 1.5), (r(2, T, H), -1.0)]]
    for terms in cases:
        total = sum(s * (t.double().sum(0) if t.dim() == 3 else t.double()) for t, s in terms)
        ref = x.double() + plain.layer_norm(total, w.double(), b.double(), 1e-5)
        xd = x.to(DEV)
        y = torch.empty(T, H, dtype=out_dtype, device=DEV)
        K.add_layer_norm(xd, [(t.to(DEV).contiguous(), s) for t, s in terms], w.to(DEV), b.to(DEV), 1e-5, y=y)
        close(xd, ref, 1e-5)
        close(y, ref, 1e-5 if out_dtype == torch.float32 else 6e-3)
        xd = x.to(DEV)
        K.add_layer_norm(xd, [(t.to(DEV).contiguous(), s) for t, s in terms], w.to(DEV), b.to(DEV), 1e-5)
        close(xd, ref, 1e-5)


@pytest.mark.parametrize("T,H,dim,layers", [(1, 72, 12, 3), (9, 128, 16, 5), (300, 50, 5, 2), (8, 2304, 128, 2)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_tokens_own_row(K, T, H, dim, layers, dtype):
    """Every layer's part of the table, the gate from a product with and without split sums."""
    from airframe_b200.config.base import PartSpec
    from airframe_b200.parts import BuildContext, build_part
    from airframe_b200.parts.linear import as_terms
    g = torch.Generator().manual_seed(T + H)
    r = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16).float()
    table = r(40, layers * dim)
    ids = torch.randint(0, 40, (T,), generator=g)
    h = r(T, H)
    for i in range(layers):
        W = {"t": table, "g": r(dim, H) * H ** -0.5, "p": r(H, dim)}
        part = build_part("feed_forward", PartSpec("token_side", {
            "hidden_size": H, "dim": dim, "vocab_size": 40, "index": i, "parts": layers, "activation": "gelu_tanh",
            "table_weight": "t", "gate_weight": "g", "proj_weight": "p"}), BuildContext(compute_dtype=dtype, device=torch.device(DEV)))
        part.load({n: t.to(DEV).to(dtype) for n, t in W.items()})
        out = torch.zeros(T, H, device=DEV)
        K.add_scaled_rmsnorm(out, as_terms(part.forward(h.to(DEV).to(dtype), SimpleNamespace(tokens=i32(ids.tolist())))))
        Wd = {"side.embed": table.double(), "side.gate": W["g"].to(dtype).double(), "side.proj": W["p"].double()}
        close(out, plain.token_side(h.double(), ids.tolist(), Wd, "", i, dim), 1e-5 if dtype == torch.float32 else 1.5e-2, i)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,heads,D,N,extra", [(3, 4, 20, 14, 0), (70, 2, 40, 300, 0), (8, 3, 96, 64, 16), (65, 5, 24, 33, 4)])
@pytest.mark.parametrize("at,pad", [(3, 5), (4, 4)])
def test_a_gate_per_value(K, T, heads, D, N, extra, dtype, at, pad):
    g = torch.Generator().manual_seed(T + N)
    r = lambda *s: torch.randn(*s, generator=g)
    x, w, gate = r(T, heads, D + extra).to(dtype), r(heads, D, N).to(dtype), r(T, -(-heads * N // 4) * 4 + 8)
    out = torch.empty(T, heads * (N + extra), dtype=dtype, device=DEV)
    gd = gate.to(DEV)[:, at: at + heads * N]
    K.head_project(out, x.reshape(T, -1).to(DEV), w.to(DEV), heads, D, N, extra=extra, gate=gd)
    s = plain.sigmoid(gate[:, at: at + heads * N].double()).view(T, heads, N)
    ref = torch.einsum("thd,hdn->thn", x[..., :D].double(), w.double()) * s
    got = out.view(T, heads, N + extra).cpu()
    close(got[..., :N], ref, 1e-5 if dtype == torch.float32 else 1e-2)
    assert torch.equal(got[..., N:], x[..., D:])                              # (what is copied is not gated)
    y = r(T, heads, N + pad).to(dtype)
    yd = y.reshape(T, -1).to(DEV)
    K.head_gate(yd, gd, heads, N, per_value=True, pitch=N + pad)
    got = yd.view(T, heads, N + pad).cpu()
    close(got[..., :N], y[..., :N].double() * s, 1e-5 if dtype == torch.float32 else 1e-2)
    assert torch.equal(got[..., N:], y[..., N:])
