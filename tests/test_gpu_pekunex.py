"""Pekunex on the GPU against the plain implementation (oracle/pekunex_ref.py, float64, whole sequences, no cache):
every mechanism alone, then whole models through the engine's runner, scheduler bookkeeping and cache / state manager --
prompts, token-by-token decoding, portions, mixed batches, reused pages and slots -- and greedy generation through LLM."""
import math

import pytest
import torch

import pekunex_helpers as ph
from oracle import pekunex_ref as ref
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
def test_residual_update_and_rms_norm(dtype, cols):
    """The update, the norm and its constant factor in one pass, rows wider than a thread's registers, widths that are not multiples of
    four, small rows whose eps counts, selected rows, update alone and norm alone."""
    from nanovllm.layers.layernorm import PreNorm
    from nanovllm import mixops
    g = torch.Generator().manual_seed(cols)
    eps = 1e-2
    n = PreNorm(cols, eps, DT[dtype], "cuda", scale=0.37)
    w = (1 + 0.3 * torch.randn(cols, generator=g)).to(DT[dtype])
    n.weight.copy_(w)
    x = torch.randn(5, cols, generator=g) * torch.tensor([2.0, 0.1, 30.0, 1e-3, 1.0])[:, None]
    y = (torch.randn(5, cols, generator=g) * torch.tensor([1.0, 0.1, 1.0, 1e-3, 1.0])[:, None]).to(DT[dtype])
    want_x = x.double() + y.double()
    tol = 4e-6 if dtype == "float32" else 4e-3
    xd = x.cuda()
    out = n.after(xd, y.cuda())
    assert rel_err(xd, want_x) < 1e-6 and rel_err(out, ref.rms_norm(want_x, w, eps) * 0.37) < tol
    for r in range(5):
        assert rel_err(out[r], ref.rms_norm(want_x[r], w, eps) * 0.37) < tol, r
    before = xd.clone()
    assert torch.equal(n.open(xd), out)
    assert torch.equal(n.open(xd, torch.tensor([4, 0, 4], dtype=torch.int32, device="cuda")), out[[4, 0, 4]]) and torch.equal(xd, before)
    assert mixops.add_rmsnorm(xd, None, eps, y=y.cuda()) is None and rel_err(xd, want_x + y.double()) < 1e-6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("ff", [72, 23])
def test_silu_gated_feed_forward(dtype, ff):
    from nanovllm.layers.moe import SiluGatedDenseFF
    g = torch.Generator().manual_seed(ff)
    width = 40
    W = {"gate": torch.randn(ff, width, generator=g) * 0.4, "up": torch.randn(ff, width, generator=g) * 0.4, "down": torch.randn(width, ff, generator=g) * 0.2}
    W = {k: v.to(DT[dtype]) for k, v in W.items()}
    layer = SiluGatedDenseFF(width, {"ff": ff}, DT[dtype], "cuda")
    for k, v in W.items():
        assert layer.load(k, v)
    h = torch.randn(13, width, generator=g).to(DT[dtype])
    assert rel_err(layer.forward(h.cuda())[0], ref.dense_ff(W, "", h.double())) < (1e-5 if dtype == "float32" else 1.5e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("pad", [5, 8])
@pytest.mark.parametrize("shape", [(3, 1, 16, 24, 8), (4, 2, 64, 32, 64), (2, 2, 9, 7, 4), (5, 5, 32, 128, 0), (2, 1, 96, 16, 48), (1, 1, 200, 8, 66),
                                   (40, 4, 128, 64, 64), (3, 3, 16, 8, 16), (2, 1, 256, 24, 32), (1, 1, 48, 40, 16)])
def test_unit_norm_after_the_rotation(dtype, shape, pad):
    """Rotated part scaled by the table's magnitude, the rest not, then one root mean square over both (with an eps that counts for small
    heads); positions up to the thousands; keys cached so, values as they are; a token with slot -1 stores nothing."""
    from nanovllm import mixops
    from nanovllm.layers.rotary_embedding import build_scaled_cos_sin
    H, G, d, vd, dims = shape
    g = torch.Generator().manual_seed(sum(shape))
    n, base, eps = 9, 777.0, 1e-2
    cols = H * d + G * d + G * vd + pad                       # 5: rows that are not 16-byte aligned
    x = (torch.randn(n, cols, generator=g) * torch.tensor([1.0, 0.05, 3.0, 1.0, 0.2, 1.0, 1.0, 10.0, 1.0])[:, None]).to(DT[dtype])
    pos = torch.tensor([0, 1, 2, 63, 64, 500, 1999, 3, 1000], dtype=torch.int64)
    slots = torch.tensor([4, 0, 17, -1, 3, 9, 8, 30, 1], dtype=torch.int32)
    cache = torch.full((32, G * (d + vd)), 7.0, dtype=DT[dtype], device="cuda")
    table = build_scaled_cos_sin(dims, 2048, base, ph.RAMP, "cuda") if dims else None
    xd = x.cuda().clone()
    mixops.headnorm_rope_store(xd, 0, H * d, H * d + G * d, H, G, d, vd, None, None, False, table, pos.cuda(), slots.cuda(), cache, eps,
                               layout=mixops.ROT_HALVES, unit_after=True)

    def unit(y):
        out = y.clone()
        for t in range(n if dims else 0):
            full = torch.zeros(int(pos[t]) + 1, y.shape[1], d, dtype=F64)
            full[-1] = y[t]
            out[t] = ref.rotate_halves(full, *ref.ramp_frequencies(dims, base, ph.RAMP))[-1]
        return ref.unit_rms(out, eps)
    xx = x.double()
    tol = 3e-6 if dtype == "float32" else 4e-3
    wantq, wantk = unit(xx[:, :H * d].view(n, H, d)).reshape(n, -1), unit(xx[:, H * d:H * d + G * d].view(n, G, d)).reshape(n, -1)
    for t, s in enumerate(slots.tolist()):
        assert rel_err(xd[t, :H * d], wantq[t]) < tol, t
        if s >= 0:
            assert rel_err(cache[s, :G * d], wantk[t]) < tol and torch.equal(cache[s, G * d:].cpu(), x[t, H * d + G * d:H * d + G * d + G * vd])
    assert bool((cache[[s for s in range(32) if s not in slots.tolist()]] == 7.0).all())
    assert torch.equal(xd[:, H * d:].cpu(), x[:, H * d:])                       # only the queries change in place


def plain_heads(q, k, v, H, G, scale, cap, sinks, gate, out_scale, rows):
    """float64: soft-capped causal softmax (with the sink's term), gated element by element -> [rows, H, vd]."""
    out = []
    for h in range(H):
        s = (q[:, h] @ k[:, h // (H // G)].T) * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        P = ref.causal_softmax(s, None if sinks is None else float(sinks[h]))
        out.append(out_scale * (P @ v[:, h // (H // G)]) * (torch.sigmoid(gate[:, h]) if gate is not None else 1.0))
    return torch.stack(out, 1)[rows]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("bs,d,vd", [(16, 32, 32), (64, 48, 40), (64, 96, 72), (16, 20, 12)])
def test_capped_attention_finds_one_key_anywhere(dtype, bs, d, vd):
    """One key is made to stand out for head 1, so that half of its weight sits on it under the cap (and all of it without): at position 0,
    at page borders, far back and at the query itself; as the last row of a portion and as a decoded token; pages are scrambled and hold
    a stale row beyond the sequence's end that would take all the weight."""
    from nanovllm import mixops
    H, G, L, cap, scale = 4, 2, 330, 6.5, 0.2
    g = torch.Generator().manual_seed(bs + d)
    npages = (L + bs - 1) // bs + 1
    pages = torch.randperm(40, generator=g)[:npages]
    for star in sorted({0, 1, bs - 1, bs, 63, 64, 129, L - 2, L - 1}):
        q = torch.randn(L, H * d, generator=g) * 0.3
        k = torch.randn(L, G * d, generator=g) * 0.3
        v = torch.randn(L, G * vd, generator=g)
        gate = torch.randn(L, H * vd + 4, generator=g).to(DT[dtype])
        for pos in sorted({star, star + 1, L - 1} & set(range(star, L))):
            qq, kk = q.clone(), k.clone()
            u = qq[pos, d:2 * d] / qq[pos, d:2 * d].norm()
            kk[star, :d] = 25.0 * u                           # head 1 (key/value head 0) of position `pos` looks straight at it
            qq[pos, d:2 * d] = 8.0 * u
            stale = torch.cat([60.0 * u.repeat(G), torch.full((G * vd,), 1e3)])
            cache = paged(torch.cat([kk, v], 1), pages, bs, dtype, 40, stale=stale)
            kv = torch.stack([cache[int(pages[j // bs]) * bs + j % bs] for j in range(pos + 1)]).double()
            args = (qq.to(DT[dtype]).double()[:pos + 1].view(-1, H, d), kv[:, :G * d].reshape(-1, G, d), kv[:, G * d:].reshape(-1, G, vd), H, G, scale)
            gd = gate[:pos + 1, :H * vd].double().view(-1, H, vd)
            want = plain_heads(*args, cap, None, gd, 1.0, [pos])[0]
            assert pos < 200 or (rel_err(plain_heads(*args, 0.0, None, gd, 1.0, [pos])[0][1], want[1]) > 0.1)       # without the cap it would be another result
            bt = pages[None, :].to(torch.int32).cuda().contiguous()
            for decode in (False, True):
                for kw in PATHS:
                    first, sp = (pos, spans_decode([pos + 1])) if decode else (max(0, pos - 20), None)
                    sp = sp or spans_varlen([pos + 1 - first], [pos + 1])
                    got = mixops.window_attention(qq[first:pos + 1].to(DT[dtype]).cuda(), cache.cuda(), bt, bs, sp, H, G, d, vd, scale, softcap=cap,
                                                  gate=gate[first:pos + 1].cuda()[:, :H * vd], **kw)
                    assert rel_err(got[-1].view(H, vd), want) < (1e-4 if dtype == "float32" else 2e-2), (star, pos, decode, kw)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", [(6, 2, 64, 64), (3, 1, 8, 24), (8, 8, 48, 40), (4, 2, 96, 96), (20, 1, 128, 32), (40, 2, 80, 128), (2, 1, 24, 136), (5, 5, 9, 7)])
def test_cap_sink_gate_and_factor_over_shapes_and_batches(dtype, shape):
    """Three sequences in one step (portions behind cached tokens, and single tokens), every combination of cap, learned sinks, element gate
    and factor, head sizes the tensor-core kernel takes as they are, pads and leaves to the FMA kernel; the result lands in a column slice
    of a wider buffer."""
    from nanovllm import mixops
    H, G, d, vd = shape
    g = torch.Generator().manual_seed(sum(shape))
    lens, bs, scale = (150, 67, 5), 16, 1.5 / d ** 0.5
    pages = torch.randperm(30, generator=g)
    used, seqs = 0, []
    tables = torch.full((3, 10), -1, dtype=torch.int32)
    cache = torch.full((30 * bs, G * (d + vd)), 50.0, dtype=DT[dtype])
    for i, L in enumerate(lens):
        q, kv = torch.randn(L, H * d, generator=g).to(DT[dtype]), torch.randn(L, G * (d + vd), generator=g).to(DT[dtype])
        gate = (3 * torch.randn(L, H * vd, generator=g)).to(DT[dtype])
        pg = pages[used:used + (L + bs - 1) // bs]
        used += len(pg)
        tables[i, :len(pg)] = pg
        for j in range(L):
            cache[int(pg[j // bs]) * bs + j % bs] = kv[j]
        seqs.append((q, kv, gate))
    cache, bt = cache.cuda(), tables.cuda()
    tol = 1e-4 if dtype == "float32" else 2e-2
    results = []
    for cap, sinks, gated, factor in ((2.0, None, True, 1.0), (0.0, torch.linspace(-2, 4, H), False, 0.6), (1.5, torch.linspace(-2, 2, H), True, 1.7)):
        want = [plain_heads(q.double().view(-1, H, d), kv[:, :G * d].double().reshape(-1, G, d), kv[:, G * d:].double().reshape(-1, G, vd), H, G, scale, cap,
                            sinks, gate.double().view(-1, H, vd) if gated else None, factor, slice(None)).reshape(L, -1) for (q, kv, gate), L in zip(seqs, lens)]
        results.append(want[0])
        for spans_of in ([(0, 150), (0, 67), (0, 5)], [(81, 150), (66, 67), (3, 5)], [(149, 150), (66, 67), (4, 5)], [(79, 80), (40, 41), (0, 1)]):
            decode = all(b - a == 1 for a, b in spans_of)
            qs = torch.cat([s[0][a:b] for s, (a, b) in zip(seqs, spans_of)]).cuda()
            gs = torch.cat([s[2][a:b] for s, (a, b) in zip(seqs, spans_of)]).cuda() if gated else None
            sp = spans_decode([b for _, b in spans_of]) if decode else spans_varlen([b - a for a, b in spans_of], [b for _, b in spans_of])
            exp = torch.cat([w[a:b] for w, (a, b) in zip(want, spans_of)])
            for kw in PATHS:
                wide = torch.full((qs.shape[0], H * vd + 24), 5.0, dtype=DT[dtype], device="cuda")
                mixops.window_attention(qs, cache, bt, bs, sp, H, G, d, vd, scale, softcap=cap, sinks=sinks.cuda() if sinks is not None else None, gate=gs,
                                        out=wide[:, 8:8 + H * vd], out_scale=factor, **kw)
                assert rel_err(wide[:, 8:8 + H * vd], exp) < tol, (cap, spans_of, kw)
                assert bool((wide[:, :8] == 5.0).all()) and bool((wide[:, 8 + H * vd:] == 5.0).all())
    assert rel_err(results[0], results[1]) > 10 * tol and rel_err(results[0], results[2]) > 10 * tol


def _load(layer, W, pre):
    for leaf in layer.weight_shapes(layer.width):
        assert layer.load(leaf, W[pre + leaf]), leaf
    return layer


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("layer", [ph.attention(), ph.attention(heads=1, kv_heads=1, dim=9, vdim=5, rot_dims=0, softcap=None),
                                   ph.attention(heads=8, kv_heads=2, dim=64, vdim=32, rot_dims=64, base=500.0, scale=0.125, softcap=10.0),
                                   ph.attention(heads=6, kv_heads=2, dim=72, vdim=56, rot_dims=40, scale=0.2, softcap=3.0)])
def test_capped_attention_layer(dtype, layer):
    from nanovllm.layers.window_attention import CappedGatedAttention
    width, eps, m = 40, 1e-3, layer["mixer"]
    W = ph.random_weights(ph.config([(layer, None)], width=width), 3)
    got = _load(CappedGatedAttention(width, m, eps, DT[dtype], "cuda", 512), {k: v.to(DT[dtype]) for k, v in W.items()}, "l0.mix.")
    portions_batches_and_dirty_slots(got, lambda h: ref.gated_attention(W, "l0.mix.", m, h, eps), width, dtype)


SPACES = [ph.mamba2(), ph.mamba2(heads=1, vdim=5, state=3, groups=1, conv=1, norm_groups=1), ph.mamba2(heads=4, vdim=32, state=64, groups=2, conv=5, norm_groups=8),
          ph.mamba2(heads=3, vdim=64, state=128, groups=3, conv=2, norm_groups=3), ph.mamba2(heads=2, vdim=200, state=16, groups=1, conv=9, norm_groups=1),
          ph.mamba2(heads=4, vdim=9, state=200, groups=4, conv=3, norm_groups=6), ph.mamba2(heads=8, vdim=128, state=24, groups=1, conv=4, norm_groups=1)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("layer", SPACES)
def test_state_space_layer(dtype, layer):
    from nanovllm.layers.scalar_state import StateSpaceMixer
    width, eps, m = 40, 1e-3, layer["mixer"]
    W = ph.random_weights(ph.config([(layer, None)], width=width), 4)
    got = _load(StateSpaceMixer(width, m, eps, DT[dtype], "cuda"), {k: v.to(DT[dtype]) for k, v in W.items()}, "l0.mix.")
    portions_batches_and_dirty_slots(got, lambda h: ref.mamba2(W, "l0.mix.", m, h, eps), width, dtype, tol=3e-4 if dtype == "float32" else 4e-2)


MEMORIES = [ph.right(), ph.right(heads=1, dim=5, vdim=3, gate_cap=1.0), ph.right(heads=5, dim=40, vdim=56, gate_cap=15.0), ph.right(heads=2, dim=128, vdim=64),
            ph.right(heads=2, dim=64, vdim=31, gate_cap=3.0), ph.right(heads=1, dim=256, vdim=40), ph.right(heads=3, dim=32, vdim=128, gate_cap=12.0)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("m", MEMORIES)
def test_matrix_memory_layer(dtype, m):
    from nanovllm.layers.scalar_state import MatrixMemoryMixer
    width, eps = 40, 1e-3
    W = ph.random_weights(ph.config([(ph.parallel(r=m), None)], width=width), 5)
    got = _load(MatrixMemoryMixer(width, m, eps, DT[dtype], "cuda"), {k: v.to(DT[dtype]) for k, v in W.items()}, "l0.mix.right.")
    portions_batches_and_dirty_slots(got, lambda h: ref.matrix_memory(W, "l0.mix.right.", m, h, eps), width, dtype, tol=3e-4 if dtype == "float32" else 5e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", [0, 1, 2])
def test_two_mixers_side_by_side(dtype, which):
    from nanovllm.models.pekunex import MIXERS
    layer = [ph.parallel(), ph.parallel(ph.left(heads=5, kv_heads=5, dim=7, vdim=3, rot_dims=2), ph.right(heads=1, dim=9, vdim=5), -0.4, 2.0),
             ph.parallel(ph.left(heads=4, kv_heads=1, dim=64, vdim=48, rot_dims=64, scale=0.1), ph.right(heads=4, dim=32, vdim=64), 1.0, 0.5)][which]
    width, eps, m = 40, 1e-3, layer["mixer"]
    W = ph.random_weights(ph.config([(layer, None)], width=width), 6)
    got = _load(MIXERS["parallel"](width, m, eps, DT[dtype], "cuda", 512), {k: v.to(DT[dtype]) for k, v in W.items()}, "l0.mix.")
    portions_batches_and_dirty_slots(got, lambda h: ref.side_by_side(W, "l0.mix.", m, h, eps), width, dtype, tol=3e-4 if dtype == "float32" else 4e-2)


CUTS = ([600], [599, 1], [1, 2, 3, 4, 5, 6, 7, 572], [301, 299], [63, 1, 64, 65, 2, 405], [590] + [1] * 10)


def walk(n, cuts, slot, call):
    """call(rows a..b, spans) for every portion of a sequence of n tokens cut at `cuts`."""
    outs, at = [], 0
    for c in cuts:
        sp = spans_decode([at + 1]) if c == 1 and at else spans_varlen([c], [at + c])
        outs.append(call(slice(at, at + c), sp))
        at += c
    assert at == n
    return torch.cat(outs)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim,vdim,H,G", [(24, 40, 2, 1), (64, 64, 2, 2), (128, 72, 3, 1), (200, 33, 2, 2), (128, 128, 1, 1), (16, 16, 4, 2)])
def test_state_space_states_on_long_sequences(dtype, dim, vdim, H, G):
    """600 tokens in one step or cut anywhere (also token by token, and inside a block or chunk), against the plain recurrence in float64;
    decays from nearly one to nearly zero."""
    from nanovllm import mixops
    g = torch.Generator().manual_seed(dim)
    n = 600
    x = torch.randn(n, 2 * G * dim + H * vdim, generator=g).to(DT[dtype])
    step = (torch.randn(n, H, generator=g) * 4 - 3).to(DT[dtype])
    rate, bias = -torch.linspace(1.5, 0.05, H), torch.randn(H, generator=g)
    dt = torch.nn.functional.softplus(step.double() + bias.double())
    decay = torch.exp(dt * rate.double())
    assert decay.min() < 1e-2 and decay.max() > 0.999
    v, k, q = x[:, :H * vdim].double().view(n, H, vdim), x[:, H * vdim:H * vdim + G * dim].double().view(n, G, dim), x[:, H * vdim + G * dim:].double().view(n, G, dim)
    want = torch.stack([ref.state_space(v[:, h], k[:, h // (H // G)], q[:, h // (H // G)], dt[:, h], torch.log(-rate[h]).item()) for h in range(H)], 1)
    S = torch.stack([sum(torch.exp(rate[h].double() * dt[t + 1:, h].sum()) * dt[t, h] * torch.outer(v[t, h], k[t, h // (H // G)]) for t in range(n)) for h in range(H)])
    slot = torch.zeros(1, dtype=torch.int32, device="cuda")
    xd, sd = x.cuda(), step.cuda()
    for cuts, fma in ((c, f) for c in CUTS for f in (False, True)):
        state = torch.full((1, H, vdim, dim), 9.0, device="cuda")            # a new sequence ignores what the slot holds
        out = walk(n, cuts, slot, lambda r, sp: mixops.linear_state(xd[r], H * vdim + G * dim, H * vdim, 0, state, slot, sp, H, G, dim, vdim, step=sd[r],
                                                                   rate=rate.cuda(), bias=bias.cuda(), fma=fma))
        assert rel_err(out, want) < 3e-5 and rel_err(state[0], S) < 3e-5, (cuts, fma)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim,vdim,H", [(24, 40, 2), (64, 64, 2), (128, 72, 1), (200, 33, 2), (128, 128, 1), (16, 16, 4), (32, 63, 3)])
@pytest.mark.parametrize("mood", ["mixed", "rising", "shut"])
def test_memory_cells_on_long_sequences(dtype, dim, vdim, H, mood):
    """Gates, running maximum, states and normaliser over 600 tokens, cut anywhere, against the plain recurrence: input gates that jump over
    the whole capped range, that drive the maximum up, and that stay far below it (so that exp(-m) is the larger divisor)."""
    from nanovllm import mixops
    g = torch.Generator().manual_seed(dim + vdim)
    n, cap = 600, 9.0
    x = torch.randn(n, H * (2 * dim + vdim), generator=g).to(DT[dtype])
    pre = torch.randn(n, 2 * H, generator=g) * torch.tensor([6.0] * H + [3.0] * H)
    bias = torch.cat([torch.full((H,), {"mixed": -1.0, "rising": 6.0, "shut": -20.0}[mood]), torch.linspace(1.0, 6.0, H)])
    i = cap * torch.tanh((pre[:, :H] + bias[:H]).double() / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((pre[:, H:] + bias[H:]).double() / cap))
    q, k, v = x[:, :H * dim].double().view(n, H, dim) * dim ** -0.5, x[:, H * dim:2 * H * dim].double().view(n, H, dim), x[:, 2 * H * dim:].double().view(n, H, vdim)
    want, nq, top = (torch.stack(p, 1) for p in zip(*(ref.memory_parts(q[:, h], k[:, h], v[:, h], i[:, h], f[:, h]) for h in range(H))))
    floor = torch.exp(-top)
    assert bool((nq.abs() < floor).any()) and (mood == "shut" or bool((nq.abs() > floor).any()))
    slot = torch.zeros(1, dtype=torch.int32, device="cuda")
    xd, pd = x.cuda(), pre.cuda()
    for cuts, fma in ((c, f) for c in CUTS for f in (False, True)):
        state, m = torch.full((1, H, vdim + 1, dim), 9.0, device="cuda"), torch.full((1, H), 5.0, device="cuda")

        def call(r, sp):
            ld, w, fl = mixops.mlstm_gates(pd[r], bias.cuda(), cap, m, slot, sp, H)
            o = mixops.linear_state(xd[r], 0, H * dim, 2 * H * dim, state, slot, sp, H, H, dim, vdim, dim ** -0.5, log_decay=ld, write=w, ones=True,
                                    fma=fma)
            return torch.cat([o, fl[..., None]], -1)
        o = walk(n, cuts, slot, call)                        # before the division, which amplifies the rounding of a small n . q
        assert rel_err(o[..., :vdim], want) < 5e-5 and rel_err(o[..., vdim], nq) < 5e-5 and rel_err(o[..., vdim + 1], floor) < 5e-5, (cuts, fma)
        assert rel_err(m[0], top[-1]) < 1e-5, (cuts, fma)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_memory_read_out_close(dtype):
    """Divisor by the larger of the normaliser and its floor, head norm with an eps that counts, weights per head and element, sigmoid gate, factor,
    a column slice; the shared weight of the other designs still works beside it."""
    from nanovllm import mixops
    g = torch.Generator().manual_seed(4)
    n, H, vd, eps = 11, 3, 21, 1e-2
    x, fl = torch.randn(n, H, vd + 1, generator=g) * 0.3, torch.rand(n, H, generator=g) * 0.4
    w, gate = torch.randn(H * vd, generator=g).to(DT[dtype]), torch.randn(n, H * vd + 3, generator=g).to(DT[dtype])
    o = x[..., :vd].double() / (torch.maximum(x[..., vd].double().abs(), fl.double()) + 1e-6)[..., None]
    want = 1.3 * ref.unit_rms(o, eps).reshape(n, -1) * w.double() * torch.sigmoid(gate[:, :H * vd].double())
    wide = torch.full((n, H * vd + 16), 5.0, dtype=DT[dtype], device="cuda")
    mixops.head_rmsnorm_gate(x.cuda(), w.cuda(), gate.cuda()[:, :H * vd], eps, DT[dtype], silu=False, out=wide[:, 8:8 + H * vd], out_scale=1.3, floor=fl.cuda())
    tol = 1e-5 if dtype == "float32" else 4e-3
    assert rel_err(wide[:, 8:8 + H * vd], want) < tol and bool((wide[:, :8] == 5.0).all()) and bool((wide[:, 8 + H * vd:] == 5.0).all())
    y = x[..., :vd].contiguous()
    got = mixops.head_rmsnorm_gate(y.cuda(), w[:vd].cuda(), None, eps, DT[dtype])
    assert rel_err(got, (ref.unit_rms(y.double(), eps) * w[:vd].double()).reshape(n, -1)) < tol


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,vd,groups", [(6, 10, 2), (4, 64, 4), (3, 7, 7), (32, 128, 1), (1, 5, 1), (8, 48, 3)])
def test_state_space_close(dtype, H, vd, groups):
    """Skip per head, gate BEFORE the norm, parts of the row that do not line up with the heads."""
    from nanovllm import mixops
    g = torch.Generator().manual_seed(H + vd)
    n, inner, eps = 7, H * vd, 1e-2
    y, D = torch.randn(n, H, vd, generator=g), torch.randn(H, generator=g)
    x, z, w = (torch.randn(n, inner + 12, generator=g).to(DT[dtype]), torch.randn(n, inner + 8, generator=g).to(DT[dtype]), torch.randn(inner, generator=g).to(DT[dtype]))
    t = (y.double() + D.double()[:, None] * x[:, 4:4 + inner].double().view(n, H, vd)).reshape(n, inner) * ref.silu(z[:, :inner].double())
    want = ref.unit_rms(t.view(n, groups, -1), eps).reshape(n, inner) * w.double()
    got = mixops.skip_gate_groupnorm(y.cuda(), x.cuda()[:, 4:4 + inner], D.cuda(), z.cuda()[:, :inner], w.cuda(), groups, eps)
    assert rel_err(got, want) < (1e-5 if dtype == "float32" else 4e-3)


# ---------------------------------------------------------------------------------------------------------------------------
# whole models through the engine
# ---------------------------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def checkpoints(tmp_path_factory):
    root = tmp_path_factory.mktemp("pekunex")
    out = {}
    for name, cfg in (("a", ph.config_a()), ("b", ph.config_b()), ("c", ph.config_c()), ("d", ph.config_d())):
        W = ph.random_weights(cfg, 21)
        out[name] = (ph.write_checkpoint(str(root / name), cfg, W), cfg, W)
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
    """fp32: the RMS error over everything.  bf16: in these tiny random models a token whose small query or key of a dozen elements is made a
    unit vector, or whose memory is divided by a small normaliser, can come out several times worse than its neighbours; the bound is on
    the median over positions, with a loose one on the sum."""
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
        toks = ph.tokens(n, vocab, i)
        got = e.step([("p", toks)])["p"]
        e.end("p")
        assert_logits(got, oracle_logits(checkpoints, name, toks), dtype, n)


def test_the_stream_after_every_layer(checkpoints):
    """The residual stream after each layer (borrowing ones too) against the plain implementation."""
    e = Replay(checkpoints["a"][0], "float32", eager=True)
    _, cfg, W = checkpoints["a"]
    toks = ph.tokens(45, cfg["vocab"], 3)
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
    assert len(taps) == len(want) == len(cfg["layers"])
    for r, (a, b) in enumerate(zip(taps, want)):
        assert rel_err(a, b) < 1e-4, r


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "b"])
def test_long_decoding_matches_the_prompt_path(engines, checkpoints, name, dtype):
    """One prompt token, then 170 tokens one by one through the decode graphs, across ten pages."""
    e = engines(name, dtype)
    toks = ph.tokens(171, checkpoints[name][1]["vocab"], 5)
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
    toks = ph.tokens(sum(cuts), checkpoints[name][1]["vocab"], 6)
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
    T = {k: ph.tokens(n, vocab, 10 + i) for i, (k, n) in enumerate(dict(a=90, b=37, c=9, d=140, e=70, f=44).items())}
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
    beside page borders, then single tokens, next to a second request that arrives in the middle."""
    e = Replay(checkpoints["c"][0], dtype, pool_tokens=768, block=64, seqs=3)
    vocab = checkpoints["c"][1]["vocab"]
    T = {"a": ph.tokens(333, vocab, 81), "b": ph.tokens(90, vocab, 82)}
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
    x, y = ph.tokens(50, vocab, 30), ph.tokens(21, vocab, 31)
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
    prompts = [ph.tokens(n, cfg["vocab"], 40 + i) for i, n in enumerate((5, 61, 1, 100, 18))]      # more requests than slots, chunked prompts
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
    toks = ph.tokens(40, cfg["vocab"], 50)
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
