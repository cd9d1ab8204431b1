"""Zuvepel on the GPU against the plain implementation (oracle/zuvepel_ref.py, float64, whole sequences, no cache):
every mechanism alone, then whole models through the engine's runner, scheduler bookkeeping and cache / state manager --
prompts, token-by-token decoding, portions, mixed batches, reused pages and slots -- and greedy generation through LLM."""
import math

import pytest
import torch

import zuvepel_helpers as zh
from oracle import zuvepel_ref as ref
from test_gpu_musavik import PATHS, paged, portions_batches_and_dirty_slots, run_parts, spans_decode
from test_gpu_tafopel import Replay, rel_err, spans_varlen

pytestmark = pytest.mark.gpu

DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
TOL = {"float32": 3e-4, "bfloat16": 6e-2}
F64 = torch.float64


# ---------------------------------------------------------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cols", [45, 200, 1000, 1101, 2000, 4096, 4500])
def test_two_norms_of_one_stream(dtype, cols):
    """The scaled update, the extra addend, both norms from one pair of statistics (a large common offset in the rows), rows wider than
    a thread's registers, widths that are not multiples of four, a destination other than the source, selected rows."""
    from nanovllm import mixops
    g = torch.Generator().manual_seed(cols)
    vec = lambda: (1 + 0.3 * torch.randn(cols, generator=g)).to(DT[dtype])
    n1, n2 = (vec(), vec()), (vec(), vec())
    x, add = torch.randn(5, cols, generator=g) * 2 + 30.0, torch.randn(5, cols, generator=g)
    y = torch.randn(5, cols, generator=g).to(DT[dtype])
    cu = lambda p: tuple(t.cuda() for t in p)
    tol = 4e-6 if dtype == "float32" else 4e-3
    want_x = x.double() + 0.37 * y.double() + add.double()
    xd, out = x.cuda(), torch.zeros(5, cols, device="cuda")
    a, b = mixops.add_layernorm2(xd, 1e-5, y=y.cuda(), mult=0.37, add=add.cuda(), x_out=out, norm1=cu(n1), norm2=cu(n2))
    assert torch.equal(xd.cpu(), x) and rel_err(out, want_x) < 1e-6          # the source is left alone; the stream stays fp32
    assert rel_err(a, ref.layer_norm(want_x, *n1, 1e-5)) < tol and rel_err(b, ref.layer_norm(want_x, *n2, 1e-5)) < tol
    a2, none = mixops.add_layernorm2(xd, 1e-5, y=y.cuda(), mult=0.37, norm1=cu(n2))                # in place, one norm
    assert none is None and rel_err(xd, x.double() + 0.37 * y.double()) < 1e-6
    assert rel_err(a2, ref.layer_norm(x.double() + 0.37 * y.double(), *n2, 1e-5)) < tol
    before = xd.clone()
    sel, _ = mixops.add_layernorm2(xd, 1e-5, norm1=cu(n2), rows_idx=torch.tensor([4, 0, 4], dtype=torch.int32, device="cuda"))
    assert torch.equal(sel, a2[[4, 0, 4]]) and torch.equal(xd, before)
    assert mixops.add_layernorm2(xd, 1e-5, y=y.cuda(), mult=2.0) == (None, None) and rel_err(xd, before.double().cpu() + 2 * y.double()) < 1e-6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("ff", [72, 23])
def test_gated_feed_forward_into_a_column_slice(dtype, ff):
    from nanovllm.layers.moe import GatedDenseFF
    g = torch.Generator().manual_seed(ff)
    width = 40
    W = {"gate": torch.randn(ff, width, generator=g) * 0.4, "up": torch.randn(ff, width, generator=g) * 0.4, "down": torch.randn(width, ff, generator=g) * 0.2}
    W = {k: v.to(DT[dtype]) for k, v in W.items()}
    wide = torch.zeros(width, ff + 16, dtype=DT[dtype], device="cuda")
    layer = GatedDenseFF(width, {"ff": ff}, DT[dtype], "cuda", w_down=wide[:, 16:])
    for k, v in W.items():
        assert layer.load(k, v)
    h = torch.randn(13, width, generator=g).to(DT[dtype])
    both = torch.full((13, ff + 16), 5.0, dtype=DT[dtype], device="cuda")
    layer.hidden(h.cuda(), out=both[:, 16:])
    assert bool((both[:, :16] == 5.0).all())
    tol = 1e-5 if dtype == "float32" else 1.5e-2
    want = ref.dense_ff(W, "", h.double())
    assert rel_err(both[:, 16:].double() @ wide[:, 16:].double().T, want) < tol and rel_err(layer.forward(h.cuda())[0], want) < tol


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", [(3, 1, 16, 24, 8), (4, 2, 64, 32, 64), (2, 2, 9, 7, 4), (5, 5, 32, 128, 0), (2, 1, 48, 16, 48)])
def test_half_split_rotation_and_cache_rows(dtype, shape):
    """Elements i and i + dims / 2 turn together at positions up to the thousands, the rest pass; keys are cached turned, values as
    they are; a token with slot -1 stores nothing."""
    from nanovllm import mixops
    from nanovllm.layers.rotary_embedding import build_banded_cos_sin
    H, G, d, vd, dims = shape
    g = torch.Generator().manual_seed(sum(shape))
    n, base = 9, 777.0
    cols = H * d + G * d + G * vd + 5
    x = torch.randn(n, cols, generator=g).to(DT[dtype])
    pos = torch.tensor([0, 1, 2, 63, 64, 500, 1999, 3, 1000], dtype=torch.int64)
    slots = torch.tensor([4, 0, 17, -1, 3, 9, 8, 30, 1], dtype=torch.int32)
    cache = torch.full((32, G * (d + vd)), 7.0, dtype=DT[dtype], device="cuda")
    table = build_banded_cos_sin(dims, 2048, base, None, "cuda") if dims else None
    xd = x.cuda().clone()
    mixops.headnorm_rope_store(xd, 0, H * d, H * d + G * d, H, G, d, vd, None, None, False, table, pos.cuda(), slots.cuda(), cache, 0.0,
                               layout=mixops.ROT_HALVES)

    def turned(y):
        out = y.clone()
        for t in range(n if dims else 0):
            full = torch.zeros(int(pos[t]) + 1, y.shape[1], d, dtype=F64)
            full[-1] = y[t]
            out[t] = ref.rotate_halves(full, dims, base)[-1]
        return out
    xx = x.double()
    tol = 3e-6 if dtype == "float32" else 4e-3
    assert rel_err(xd[:, :H * d], turned(xx[:, :H * d].view(n, H, d)).reshape(n, -1)) < tol
    wantk = turned(xx[:, H * d:H * d + G * d].view(n, G, d)).reshape(n, -1)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            assert rel_err(cache[s, :G * d], wantk[t]) < tol and torch.equal(cache[s, G * d:].cpu(), x[t, H * d + G * d:H * d + G * d + G * vd])
    assert bool((cache[[s for s in range(32) if s not in slots.tolist()]] == 7.0).all())
    assert torch.equal(xd[:, H * d:].cpu(), x[:, H * d:])                       # only the queries change in place


def plain_chunked(q, k, v, H, G, scale, chunk, sinks, gate, rows):
    """float64: softmax with the sink's term per head over the keys of the query's chunk, gated -> [rows, H, vd]."""
    L = k.shape[0]
    see = ref.same_chunk(L, chunk)
    out = []
    for h in range(H):
        s = (q[:, h] @ k[:, h // (H // G)].T) * scale
        s = torch.where(see, s, torch.full_like(s, -math.inf))
        p = torch.softmax(torch.cat([s, torch.full((L, 1), float(sinks[h]), dtype=F64)], 1), 1)[:, :L]
        out.append((p @ v[:, h // (H // G)]) * torch.sigmoid(gate[:, h:h + 1]))
    return torch.stack(out, 1)[rows]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("bs,chunk", [(16, 50), (64, 64), (64, 65), (16, 128), (16, 1), (64, 200), (16, 0)])
def test_attention_sees_its_own_chunk_only(dtype, bs, chunk):
    """One key is made to dominate head 1: the head's weight must sit on it exactly while the query is in the key's chunk.  The key
    sits at the start, in the middle and at the last place of a chunk, at page borders and far back; the query is the last place of
    that chunk, the first of the next, a later one, as the last row of a portion and as a decoded token; pages are scrambled and hold
    a stale dominating row beyond the sequence's end."""
    from nanovllm import mixops
    H, G, d, vd, L = 4, 2, 32, 32, 330
    g = torch.Generator().manual_seed(bs + chunk)
    npages = (L + bs - 1) // bs + 1
    pages = torch.randperm(40, generator=g)[:npages]
    size = chunk or L
    sinks = torch.zeros(H)
    for star in sorted({0, 1, size - 1, size, size + 1, 2 * size - 1, bs - 1, bs, 129, L - 2} & set(range(L - 1))):
        end = (star // size + 1) * size
        q = torch.randn(L, H * d, generator=g)
        k = torch.randn(L, G * d, generator=g) * 0.3
        v = torch.randn(L, G * vd, generator=g)
        gate = torch.randn(L, 8, generator=g).to(DT[dtype])
        for pos in sorted({star, star + 1, end - 1, end, end + 1, L - 1} & set(range(star, L))):
            qq, kk = q.clone(), k.clone()
            u = qq[pos, d:2 * d] / qq[pos, d:2 * d].norm()
            kk[star, :d] = 40.0 * u                           # head 1 (key/value head 0) of position `pos` looks straight at it
            qq[pos, d:2 * d] = 8.0 * u
            stale = torch.cat([60.0 * u.repeat(G), torch.full((G * vd,), 1e3)])
            cache = paged(torch.cat([kk, v], 1), pages, bs, dtype, 40, stale=stale)
            kv = torch.stack([cache[int(pages[j // bs]) * bs + j % bs] for j in range(pos + 1)]).double()
            qd = qq.to(DT[dtype]).double()
            want = plain_chunked(qd[:pos + 1].view(-1, H, d), kv[:, :G * d].reshape(-1, G, d), kv[:, G * d:].reshape(-1, G, vd), H, G, 0.2, chunk,
                                 sinks, gate[:pos + 1].double(), [pos])[0]
            far = kv[star, G * d:G * d + vd] * torch.sigmoid(gate[pos, 1].double())
            assert ((want[1] - far).abs().max().item() < 1e-3) == (pos < end), (star, pos)     # the test itself distinguishes the two cases
            bt = pages[None, :].to(torch.int32).cuda().contiguous()
            for decode in (False, True):
                for kw in PATHS:
                    if decode:
                        first, sp = pos, spans_decode([pos + 1])
                    else:
                        first = max(0, pos - 20)
                        sp = spans_varlen([pos + 1 - first], [pos + 1])
                    got = mixops.window_attention(qq[first:pos + 1].to(DT[dtype]).cuda(), cache.cuda(), bt, bs, sp, H, G, d, vd, 0.2, chunk=chunk,
                                                  sinks=sinks.cuda(), gate=gate[first:pos + 1].cuda()[:, :H], **kw)
                    assert rel_err(got[-1].view(H, vd), want) < (1e-4 if dtype == "float32" else 2e-2), (star, pos, decode, kw)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", [(6, 2, 64, 64), (3, 1, 8, 24), (8, 8, 32, 32), (4, 2, 48, 40), (20, 1, 128, 32), (40, 2, 32, 128)])
def test_sink_and_head_gates_over_shapes_and_batches(dtype, shape):
    """Three sequences in one step (portions behind cached tokens, and single tokens): small scores, so that the sink takes most of a
    chunk's first rows and a fair part of all; sinks of other scores than zero; gates from nearly shut to open; the result lands in a
    column slice of a wider buffer."""
    from nanovllm import mixops
    H, G, d, vd = shape
    g = torch.Generator().manual_seed(sum(shape))
    lens, bs, chunk, scale = (150, 67, 5), 16, 40, 0.5 / d ** 0.5
    pages = torch.randperm(30, generator=g)
    used, seqs = 0, []
    tables = torch.full((3, 10), -1, dtype=torch.int32)
    cache = torch.zeros(30 * bs, G * (d + vd), dtype=DT[dtype])
    for i, L in enumerate(lens):
        q, kv = torch.randn(L, H * d, generator=g).to(DT[dtype]), torch.randn(L, G * (d + vd), generator=g).to(DT[dtype])
        gate = (3 * torch.randn(L, H, generator=g)).to(DT[dtype])
        pg = pages[used:used + (L + bs - 1) // bs]
        used += len(pg)
        tables[i, :len(pg)] = pg
        for j in range(L):
            cache[int(pg[j // bs]) * bs + j % bs] = kv[j]
        seqs.append((q, kv, gate))
    cache, bt = cache.cuda(), tables.cuda()
    tol = 1e-4 if dtype == "float32" else 2e-2
    for sinks in (torch.zeros(H), torch.linspace(-3, 3, H)):
        want = [plain_chunked(q.double().view(-1, H, d), kv[:, :G * d].double().reshape(-1, G, d), kv[:, G * d:].double().reshape(-1, G, vd), H, G,
                              scale, chunk, sinks, gate.double(), slice(None)).reshape(L, -1) for (q, kv, gate), L in zip(seqs, lens)]
        for spans_of in ([(0, 150), (0, 67), (0, 5)], [(81, 150), (66, 67), (3, 5)], [(149, 150), (66, 67), (4, 5)], [(79, 80), (40, 41), (0, 1)]):
            decode = all(b - a == 1 for a, b in spans_of)
            qs = torch.cat([s[0][a:b] for s, (a, b) in zip(seqs, spans_of)]).cuda()
            gs = torch.cat([s[2][a:b] for s, (a, b) in zip(seqs, spans_of)]).cuda()
            sp = spans_decode([b for _, b in spans_of]) if decode else spans_varlen([b - a for a, b in spans_of], [b for _, b in spans_of])
            exp = torch.cat([w[a:b] for w, (a, b) in zip(want, spans_of)])
            for kw in PATHS:
                wide = torch.full((qs.shape[0], H * vd + 24), 5.0, dtype=DT[dtype], device="cuda")
                mixops.window_attention(qs, cache, bt, bs, sp, H, G, d, vd, scale, chunk=chunk, sinks=sinks.cuda(), gate=gs, out=wide[:, 8:8 + H * vd], **kw)
                assert rel_err(wide[:, 8:8 + H * vd], exp) < tol, (spans_of, kw)
                assert bool((wide[:, :8] == 5.0).all()) and bool((wide[:, 8 + H * vd:] == 5.0).all())
    # leaving the sink out, or a gate, would show
    no_sink = plain_chunked(seqs[0][0].double().view(-1, H, d), seqs[0][1][:, :G * d].double().reshape(-1, G, d),
                            seqs[0][1][:, G * d:].double().reshape(-1, G, vd), H, G, scale, chunk, torch.full((H,), -1e9), seqs[0][2].double(), slice(None))
    assert rel_err(no_sink.reshape(150, -1), want[0]) > 10 * tol


def _load(layer, W, pre):
    for leaf in layer.weight_shapes(layer.width):
        assert layer.load(leaf, W[pre + leaf]), leaf
    return layer


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("m", [zh.attention(), zh.attention(heads=1, kv_heads=1, dim=9, vdim=5, chunk=1, rot_dims=0),
                               zh.attention(heads=8, kv_heads=2, dim=64, vdim=32, chunk=48, rot_dims=64, base=500.0, scale=0.125),
                               zh.attention(heads=6, kv_heads=2, dim=32, vdim=64, chunk=0, rot_dims=16, scale=0.2)])
def test_chunked_attention_layer(dtype, m):
    from nanovllm.layers.window_attention import ChunkedSinkAttention
    width, m = 40, m["mixer"]
    cfg = zh.config([({"type": "attention", "mixer": m}, None)], width=width)
    W = zh.random_weights(cfg, 3)
    layer = _load(ChunkedSinkAttention(width, m, 1e-5, DT[dtype], "cuda", 512), {k: v.to(DT[dtype]) for k, v in W.items()}, "l0.mix.")
    portions_batches_and_dirty_slots(layer, lambda h: ref.attention(W, "l0.mix.", m, h), width, dtype)


DELTAS = [zh.delta(), zh.delta(heads=1, kv_heads=1, dim=10, vdim=6, conv=1), zh.delta(heads=6, kv_heads=2, dim=20, vdim=40, conv=5),
          zh.delta(heads=2, kv_heads=1, dim=128, vdim=64, conv=2), zh.delta(heads=2, kv_heads=2, dim=64, vdim=33, conv=3),
          zh.delta(heads=2, kv_heads=2, dim=32, vdim=96, conv=4), zh.delta(heads=1, kv_heads=1, dim=200, vdim=36, conv=9)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("m", DELTAS)
def test_channel_delta_layer(dtype, m):
    from nanovllm.layers.channel_state import ChannelDeltaMixer
    width, eps, m = 40, 1e-5, m["mixer"]
    cfg = zh.config([({"type": "channel_delta", "mixer": m}, None)], width=width)
    W = zh.random_weights(cfg, 4)
    layer = _load(ChannelDeltaMixer(width, m, eps, DT[dtype], "cuda", ranks=zh.RANKS), {k: v.to(DT[dtype]) for k, v in W.items()}, "l0.mix.")
    portions_batches_and_dirty_slots(layer, lambda h: ref.channel_delta(W, "l0.mix.", m, h, eps), width, dtype,
                                     tol=3e-4 if dtype == "float32" else 4e-2)


GLAS = [zh.gla(), zh.gla(heads=1, dim=7, vdim=3, tau=1.0), zh.gla(heads=5, dim=40, vdim=56, tau=12.0), zh.gla(heads=2, dim=128, vdim=80, tau=2.5),
        zh.gla(heads=2, dim=64, vdim=33, tau=4.0), zh.gla(heads=1, dim=256, vdim=40, tau=8.0)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("m", GLAS)
def test_gated_linear_attention_layer(dtype, m):
    from nanovllm.layers.channel_state import GatedLinearAttention
    width, eps, m = 40, 1e-5, m["mixer"]
    cfg = zh.config([({"type": "gla", "mixer": m}, None)], width=width)
    W = zh.random_weights(cfg, 5)
    layer = _load(GatedLinearAttention(width, m, eps, DT[dtype], "cuda", ranks=zh.RANKS), {k: v.to(DT[dtype]) for k, v in W.items()}, "l0.mix.")
    portions_batches_and_dirty_slots(layer, lambda h: ref.gla(W, "l0.mix.", m, h, eps), width, dtype, tol=3e-4 if dtype == "float32" else 4e-2)


def _state_args(H, d, vd, n, g, extreme=False):
    x = torch.randn(n, 2 * H * d + H * vd, generator=g)
    z = torch.randn(n, H * d, generator=g) * (6.0 if extreme else 1.5)
    return x.cuda(), z.cuda(), torch.randn(H * d, generator=g).cuda(), -torch.rand(H, generator=g).cuda() - 0.05


@pytest.mark.parametrize("delta", [True, False])
@pytest.mark.parametrize("dim", [24, 64, 128])
def test_state_forms_agree_on_long_sequences(delta, dim):
    """600 tokens in one step or cut anywhere (also token by token, and inside a block of four), against the plain recurrence in
    float64; decays from nearly one to nearly zero."""
    from nanovllm import mixops
    H, vd, n = 2, 40, 600
    g = torch.Generator().manual_seed(dim)
    x, z, bias, rate = _state_args(H, dim, vd, n, g, extreme=True)
    write = torch.randn(n, H, generator=g).cuda() if delta else None
    sign = 1.0 if delta else -1.0
    slot = torch.zeros(1, dtype=torch.int32, device="cuda")

    def run(cuts):
        state = torch.full((1, H, vd, dim), 9.0, device="cuda")
        outs, at = [], 0
        for c in cuts:
            sp = spans_decode([at + 1]) if c == 1 and at else spans_varlen([c], [at + c])
            outs.append(mixops.channel_state(x[at:at + c], 0, H * dim, 2 * H * dim, write[at:at + c] if delta else None, z[at:at + c].clone(), rate, bias,
                                             sign, state, slot, sp, H, H, dim, vd, dim ** -0.5))
            at += c
        assert at == n
        return torch.cat(outs), state
    decay = torch.exp(rate.double().cpu()[None, :, None] * torch.nn.functional.softplus(sign * (z + bias).double().cpu().view(n, H, dim)))
    assert decay.min() < 1e-3 and decay.max() > 0.97
    q, k = (x[:, i * H * dim:(i + 1) * H * dim].double().cpu().view(n, H, dim) for i in (0, 1))
    v = x[:, 2 * H * dim:].double().cpu().view(n, H, vd)
    if delta:
        q, k = (t / torch.sqrt((t * t).sum(-1, keepdim=True) + 1e-6) for t in (q, k))
    want, S = torch.empty(n, H, vd, dtype=F64), torch.zeros(H, dim, vd, dtype=F64)
    for t in range(n):
        S = decay[t][:, :, None] * S
        u = torch.sigmoid(write[t].double().cpu())[:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t])) if delta else v[t]
        S = S + k[t][:, :, None] * u[:, None, :]
        want[t] = torch.einsum("hdv,hd->hv", S, q[t]) * dim ** -0.5
    for cuts in ([n], [n - 1, 1], [1, 2, 3, 4, 5, 6, 7, 572], [301, 299], [590] + [1] * 10):
        o, st = run(cuts)
        assert rel_err(o, want) < 2e-5 and rel_err(st[0].transpose(1, 2), S) < 2e-5, cuts


@pytest.mark.parametrize("delta", [True, False])
def test_every_key_channel_forgets_at_its_own_rate(delta):
    """One write under a key spread over all channels, then silence: reading channel by channel, what is left after 298 steps is each
    channel's own decay to that power -- half of them remember, half forget at once -- in a prompt and token by token."""
    from nanovllm import mixops
    d, vd, n = 16, 32, 300
    g = torch.Generator().manual_seed(3)
    q, k, v = torch.zeros(n, d), torch.zeros(n, d), torch.zeros(n, vd)
    k[0], v[0] = 1.0, torch.randn(vd, generator=g)
    for t in range(1, n):
        q[t, t % d] = 1.0
    x = torch.cat([q, k, v], 1).cuda()
    want_g = torch.tensor([0.999 - 0.0004 * i if i % 2 == 0 else 1e-4 for i in range(d)], dtype=F64)
    z = torch.log(torch.expm1(-torch.log(want_g))).float()[None].repeat(n, 1).cuda()       # softplus(z) = -log g, rate -1
    write = torch.full((n, 1), 40.0, device="cuda")
    args = (torch.tensor([-1.0], device="cuda"), torch.zeros(d, device="cuda"), 1.0)
    slot = torch.zeros(1, dtype=torch.int32, device="cuda")
    for cut in (n, 150):
        state = torch.full((1, 1, vd, d), 3.0, device="cuda")            # a new sequence ignores what the slot holds
        out = [mixops.channel_state(x[a:a + c], 0, d, 2 * d, write[a:a + c] if delta else None, z[a:a + c].clone(), *args, state, slot, sp, 1, 1, d, vd, 1.0)
               for a, c, sp in [(0, cut, spans_varlen([cut], [cut]))] + [(t, 1, spans_decode([t + 1])) for t in range(cut, n)]]
        out = torch.cat(out)[:, 0].double().cpu()
        scale = 0.25 if delta else 1.0                                   # the unit key of sixteen ones
        for t in (1, 2, 17, 18, 297, 298, 299):
            c = t % d
            exp = v[0].double() * scale * want_g[c] ** t
            assert (out[t] - exp).abs().max().item() < 2e-4, (cut, t)
        assert out[298].abs().max() > 0.1 * v[0].abs().max() * scale and out[299].abs().max() < 1e-6


def test_the_delta_rule_corrects_along_decayed_rows():
    """With beta = 1 a key's second value replaces what is left of the first (not its undecayed self): the read-out is exactly the
    new value; an orthogonal key's value only decays."""
    from nanovllm import mixops
    d, vd = 8, 32
    k1, k2 = torch.zeros(d), torch.zeros(d)
    k1[0], k2[3] = 1.0, 1.0
    g = torch.Generator().manual_seed(2)
    v = torch.randn(4, vd, generator=g)
    x = torch.cat([torch.stack([k1, k2, k1, k2]), torch.stack([k1, k2, k1, k1]), v], 1).cuda()
    z = torch.zeros(4, d, device="cuda")                                  # softplus(0) = ln 2, rate -1: every channel halves
    state = torch.full((1, 1, vd, d), 3.0, device="cuda")
    out = mixops.channel_state(x, 0, d, 2 * d, torch.full((4, 1), 40.0, device="cuda"), z, torch.tensor([-1.0], device="cuda"),
                               torch.zeros(d, device="cuda"), 1.0, state, torch.zeros(1, dtype=torch.int32, device="cuda"), spans_varlen([4], [4]),
                               1, 1, d, vd, 1.0)[:, 0].cpu()
    assert rel_err(out[0], v[0]) < 1e-5 and rel_err(out[1], v[1]) < 1e-5
    assert rel_err(out[2], v[2]) < 1e-5
    assert rel_err(out[3], v[1] / 4) < 1e-5                               # two halvings after its write


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["attention", "channel_delta", "gla"])
@pytest.mark.parametrize("ff", [40, 23, None])
def test_parallel_branches_share_one_output_projection(dtype, kind, ff):
    from nanovllm.layers.parallel_block import ParallelBranches
    from nanovllm.models.zuvepel import MIXERS
    width, eps = 48, 1e-5
    layer = {"attention": zh.attention(), "channel_delta": zh.delta(), "gla": zh.gla()}[kind]
    mlp = zh.dense(ff) if ff else None
    W = zh.random_weights(zh.config([(layer, mlp)], width=width), 8)
    extra = dict(max_position=256) if kind == "attention" else dict(ranks=zh.RANKS)
    b = ParallelBranches(width, MIXERS[kind], layer["mixer"], mlp, DT[dtype], "cuda", eps=eps, **extra)
    for leaf in b.mixer.weight_shapes(width):
        assert b.mixer.load(leaf, W["l0.mix." + leaf])
    for leaf in b.ff.weight_shapes(width) if ff else ():
        assert b.ff.load(leaf, W["l0.mlp." + leaf])
    b.mixer.bind(8, 16, 2, 1)
    g = torch.Generator().manual_seed(1)
    h1, h2 = torch.randn(30, width, generator=g).to(DT[dtype]), torch.randn(30, width, generator=g).to(DT[dtype])

    class Whole:                                          # run_parts drives anything with the mixers' call signature
        dtype = b.dtype

        @staticmethod
        def forward(h, pos, ctx, sp, inst):
            return b.forward(h, h2.cuda(), pos, ctx, sp, inst)
    got = run_parts(Whole, [(h1, 0, 1, [3, 0])], 16)[0]
    m = layer["mixer"]
    want = {"attention": lambda: ref.attention(W, "l0.mix.", m, h1.double()), "channel_delta": lambda: ref.channel_delta(W, "l0.mix.", m, h1.double(), eps),
            "gla": lambda: ref.gla(W, "l0.mix.", m, h1.double(), eps)}[kind]()
    if ff:
        want = want + ref.dense_ff(W, "l0.mlp.", h2.double())
    assert rel_err(got, want) < (1e-4 if dtype == "float32" else 3e-2)


# ---------------------------------------------------------------------------------------------------------------------------
# whole models through the engine
# ---------------------------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def checkpoints(tmp_path_factory):
    root = tmp_path_factory.mktemp("zuvepel")
    out = {}
    for name, cfg in (("a", zh.config_a()), ("b", zh.config_b()), ("c", zh.config_c()), ("d", zh.config_d())):
        W = zh.random_weights(cfg, 21)
        out[name] = (zh.write_checkpoint(str(root / name), cfg, W), cfg, W)
    return out


@pytest.fixture(scope="module")
def engines(checkpoints):
    made = {}

    def get(name, dtype):
        if (name, dtype) not in made:
            made[(name, dtype)] = Replay(checkpoints[name][0], dtype)
        return made[(name, dtype)]
    yield get
    for e in made.values():
        e.runner.exit()


_ORACLE: dict = {}


def oracle_logits(checkpoints, name, toks):
    key = (name, tuple(toks))
    if key not in _ORACLE:
        _, cfg, W = checkpoints[name]
        _ORACLE[key] = ref.forward(cfg, W, toks)
    return _ORACLE[key]


def assert_logits(got, want, dtype, tag=None):
    """fp32: the RMS error over everything.  bf16: a token whose small query or key of a dozen elements is then made a unit vector
    can come out several times worse than its neighbours in these tiny random models; the bound is on the median over positions,
    with a loose one on the sum."""
    got, want = got.double().cpu(), want.double().cpu()
    if dtype == "float32":
        assert rel_err(got, want) < TOL[dtype], (tag, rel_err(got, want))
    else:
        per_pos = ((got - want) ** 2).mean(1).sqrt() / (want ** 2).mean(1).sqrt()
        assert per_pos.median().item() < TOL[dtype] and rel_err(got, want) < 0.3, (tag, per_pos.median().item(), rel_err(got, want))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "b", "c", "d"])
def test_whole_prompt_and_first_tokens(engines, checkpoints, name, dtype):
    e = engines(name, dtype)
    vocab = checkpoints[name][1]["vocab"]
    for i, n in enumerate((1, 2, 17, 150)):
        toks = zh.tokens(n, vocab, i)
        got = e.step([("p", toks)])["p"]
        e.end("p")
        assert_logits(got, oracle_logits(checkpoints, name, toks), dtype, n)


def test_the_stream_after_every_layer_run(checkpoints):
    """The residual stream after each run of each layer (repeated layers count every time, before the embedding output is added)
    against the plain implementation."""
    e = Replay(checkpoints["a"][0], "float32", eager=True)
    _, cfg, W = checkpoints["a"]
    toks = zh.tokens(45, cfg["vocab"], 3)
    want = []
    ref.forward(cfg, W, toks, want)
    model, taps = e.runner.model, []
    plain_forward = model.forward
    type(model).__call__ = lambda self, ids, pos: plain_forward(ids, pos, taps)
    try:
        tapped = e.step([("p", toks)])["p"]
    finally:
        type(model).__call__ = type(model).forward
    e.end("p")
    assert rel_err(e.step([("q", toks)])["q"], tapped) < 1e-5                # collecting the stream changes nothing
    e.runner.exit()
    assert len(taps) == len(want) == 1 + 3 * 3 + 1
    for r, (a, b) in enumerate(zip(taps, want)):
        assert rel_err(a, b) < 1e-4, r


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "b"])
def test_long_decoding_matches_the_prompt_path(engines, checkpoints, name, dtype):
    """One prompt token, then 170 tokens one by one through the decode graphs, across ten pages and many chunks."""
    e = engines(name, dtype)
    toks = zh.tokens(171, checkpoints[name][1]["vocab"], 5)
    want = oracle_logits(checkpoints, name, toks)
    got = [e.step([("d", toks[:1])])["d"]]
    for t in toks[1:]:
        got.append(e.step([("d", [t])])["d"])
    e.end("d")
    got = torch.cat(got)
    assert_logits(got, want, dtype)
    assert_logits(got[-20:], want[-20:], dtype, "far end")   # no drift at the far end


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "b", "c", "d"])
def test_portions_of_many_sizes(engines, checkpoints, name, dtype):
    e = engines(name, dtype)
    cuts = (2, 3, 2, 31, 16, 2, 1, 1, 48, 15, 1, 5, 33)
    toks = zh.tokens(sum(cuts), checkpoints[name][1]["vocab"], 6)
    got, at = [], 0
    for n in cuts:
        got.append(e.step([("c", toks[at:at + n])])["c"])
        at += n
    e.end("c")
    assert_logits(torch.cat(got), oracle_logits(checkpoints, name, toks), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "b"])
def test_unequal_requests_in_one_batch_and_reused_pages_and_slots(engines, checkpoints, name, dtype):
    """Four requests of unequal length, portions beside single tokens; two of them end early and a fifth and sixth take over
    their pages and state slots while the others go on.  Every request must come out as if it had run alone."""
    e = engines(name, dtype)
    vocab = checkpoints[name][1]["vocab"]
    T = {k: zh.tokens(n, vocab, 10 + i) for i, (k, n) in enumerate(dict(a=90, b=37, c=9, d=140, e=70, f=44).items())}
    plan = [
        [("a", 40), ("b", 2)], [("a", 1), ("b", 30), ("c", 9)], [("a", 1), ("b", 1), ("d", 64)], [("a", 1), ("b", 1), ("d", 1)],
        [("a", 17), ("b", 3), ("d", 2)], [("a", 1), ("d", 1)], [("a", 29), ("d", 72)],
        # b and c are done: e and f arrive in their places
        [("e", 33), ("f", 1), ("d", 0)], [("e", 1), ("f", 43)], [("e", 36)],
    ]
    got, at, ended = {k: [] for k in T}, {k: 0 for k in T}, set()
    for step in plan:
        entries = [(k, T[k][at[k]:at[k] + n]) for k, n in step if n]
        for k, n in step:
            at[k] += n
        for k, lg in e.step(entries).items():
            got[k].append(lg)
        for k in T:
            if at[k] == len(T[k]) and k in e.live and k not in ended:
                e.end(k)
                ended.add(k)
    assert ended == set(T)
    for k in T:
        assert_logits(torch.cat(got[k]), oracle_logits(checkpoints, name, T[k]), dtype, k)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_wider_model_over_64_token_pages(checkpoints, dtype):
    """The configuration with tensor-core head sizes over pages as long as the key tile: a 333-token prompt in portions that end
    beside page and chunk borders, then single tokens, next to a second request that arrives in the middle."""
    e = Replay(checkpoints["c"][0], dtype, pool_tokens=768, block=64, seqs=3)
    vocab = checkpoints["c"][1]["vocab"]
    T = {"a": zh.tokens(333, vocab, 81), "b": zh.tokens(90, vocab, 82)}
    got, at = {"a": [], "b": []}, {"a": 0, "b": 0}
    for step in ([("a", 63)], [("a", 2)], [("a", 64), ("b", 1)], [("a", 1), ("b", 70)], [("a", 130), ("b", 1)], [("a", 1), ("b", 18)], [("a", 60)],
                 *[[("a", 1)] for _ in range(12)]):
        entries = [(k, T[k][at[k]:at[k] + n]) for k, n in step]
        for k, n in step:
            at[k] += n
        for k, lg in e.step(entries).items():
            got[k].append(lg)
    e.runner.exit()
    assert at == {"a": 333, "b": 90}
    for k, toks in T.items():
        assert_logits(torch.cat(got[k]), oracle_logits(checkpoints, "c", toks), dtype, k)


def test_batch_does_not_change_a_request_beyond_rounding(engines, checkpoints):
    e = engines("a", "float32")
    vocab = checkpoints["a"][1]["vocab"]
    x, y = zh.tokens(50, vocab, 30), zh.tokens(21, vocab, 31)
    alone = e.step([("x", x)])["x"]
    e.end("x")
    both = e.step([("y", y), ("x", x)])["x"]
    e.end("x"), e.end("y")
    assert rel_err(both, alone) < 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "d"])
def test_greedy_generation_through_the_engine(checkpoints, name, dtype):
    """LLM.generate on a checkpoint without a tokenizer: scheduler, block and slot manager, decode graphs, sampler; the attention-only
    model also skips a cached prefix.  Teacher-forced against the plain implementation: each generated token is its argmax, or
    loses to it by less than the format's rounding."""
    from nanovllm import LLM, SamplingParams
    path, cfg, W = checkpoints[name]
    llm = LLM(path, dtype=dtype, max_num_seqs=3, max_model_len=256, max_num_batched_tokens=96, kvcache_block_size=16,
              num_kvcache_blocks=24, gpu_memory_utilization=0.5)
    prompts = [zh.tokens(n, cfg["vocab"], 40 + i) for i, n in enumerate((5, 61, 1, 100, 18))]      # more requests than slots, chunked prompts
    prompts.append(prompts[3][:64] + prompts[0])                                                   # shares four pages with an earlier one
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True), use_tqdm=False)
    llm.exit()
    assert [len(o["token_ids"]) for o in outs] == [24] * 6
    tol = 1e-3 if dtype == "float32" else 0.15
    for p, o in zip(prompts, outs):
        lg = ref.forward(cfg, W, (p + o["token_ids"])[:-1])
        for i, tok in enumerate(o["token_ids"]):
            row = lg[len(p) - 1 + i]
            assert (row.max() - row[tok]).item() <= tol * row.std().item(), (len(p), i)


def test_replay_command_line(checkpoints, tmp_path):
    """bin/trace_run end to end: JSON steps on stdin, logits files and 'done' lines out."""
    import json
    import os
    import subprocess
    import numpy as np
    path, cfg, W = checkpoints["b"]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    toks = zh.tokens(40, cfg["vocab"], 50)
    steps = [{"step": 0, "entries": [{"id": "q", "tokens": toks[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "q", "tokens": toks[30:31], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "q", "tokens": toks[31:32], "want": [0]}, {"id": "r", "tokens": toks[:3], "want": [2]}], "end": ["r"]},
             {"step": 3, "entries": [{"id": "q", "tokens": toks[32:], "want": [7]}], "end": ["q"]}]
    out = tmp_path / "out"
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", str(out), "--max-tokens", "128"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    want = ref.forward(cfg, W, toks)
    rd = lambda i: torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"]))
    assert not (out / "1.f32").exists()
    assert rel_err(rd(0), want[[0, 29]]) < 3e-4 and rel_err(rd(2), torch.stack([want[31], want[2]])) < 3e-4 and rel_err(rd(3), want[[39]]) < 3e-4
