"""Each mechanism of the Nuforax layers alone, through the C ABI, against the plain implementation in tests/nuforax_plain.py (float64)."""
import ctypes as C

import numpy as np
import pytest

import nuforax_plain as npl
import sonuzen_plain as sp
from conftest import load_pkg
from device_data import EPS, Dev, pad8, rel, weights

pytestmark = pytest.mark.gpu
pkg = load_pkg()


def nans(d, nbytes):
    return d.up(np.full(max(int(nbytes), 16), 0xFF, np.uint8))


# ---- embedding and norms ---------------------------------------------------------------------

@pytest.mark.parametrize("width,buckets,mul_prev,mul_cur,cuts", [(64, 97, 31, 11, [9]), (72, 5, 4000000007, 4294967295, [1] * 6), (76, 1, 0, 3, [2, 1, 4]),
                                                                 (2056, 1000, 1, 1, [3, 3]), (30, 12, 5, 0, [1, 5])])
def test_pairs_of_tokens_and_norms_behind_sublayers(gpu, width, buckets, mul_prev, mul_cur, cuts):
    rng = np.random.default_rng(width)
    T, vocab, scale = sum(cuts), 40, 2.7
    embed, pair = weights(rng, vocab, width, scale=1.0), weights(rng, buckets + 1, width, scale=1.0)
    ids = rng.integers(0, vocab, T)
    post, last = rng.standard_normal((2, width)).astype(np.float32)
    y = rng.standard_normal((T, width)).astype(np.float32)
    x0 = embed[ids].astype(np.float64) * scale + pair[npl.bigram_rows(list(ids), buckets, mul_prev, mul_cur)]
    x1 = x0 + sp.norm_plain(y.astype(np.float64), post.astype(np.float64), EPS)
    want = sp.norm_plain(x1, last.astype(np.float64), EPS)
    with Dev(gpu) as d:
        log, demb, dpair, dpost, dlast = d.u32(ids), d.bf16(embed), d.bf16(pair), d.f32(post), d.f32(last)
        at = 0
        for n in cuts:
            pos = d.u32([at] * 4)
            xa, xb, out, trace = (d.zeros(n * pad8(width) * 4) for _ in range(4))
            a = pkg.NormConvArgs(embed=demb.value, embed_ld=pad8(width), vocab=vocab, token_log=log.value, pos=pos.value, eps=EPS, mult=1.0, x_out=xa.value, out=out.value,
                                 out_type=pkg.TYPE_F32, out_ld=pad8(width), width=width, batch=n, plain_w=1, embed_scale=scale, pair_embed=dpair.value,
                                 pair_ld=pad8(width), pair_buckets=buckets, pair_mul_prev=mul_prev, pair_mul_cur=mul_cur)
            d.call("lv_norm_conv", C.byref(a))
            assert rel(d.get(xa, (n, width)), x0[at:at + n]) < 1e-6
            assert np.array_equal(d.get(out, (n, pad8(width)))[:, :width], d.get(xa, (n, width)))       # no norm in front: the stream itself
            b = pkg.NormConvArgs(x=xa.value, y=d.f32(y[at:at + n]).value, y_rows=1, pos=pos.value, eps=EPS, mult=1.0, post_w=dpost.value, pre_w=dlast.value, x_out=xb.value,
                                 trace=trace.value, out=out.value, out_type=pkg.TYPE_F32, out_ld=pad8(width), width=width, batch=n, plain_w=1)
            d.call("lv_norm_conv", C.byref(b))
            assert rel(d.get(xb, (n, width)), x1[at:at + n]) < 1e-6 and rel(d.get(trace, (n, width)), x1[at:at + n]) < 1e-6
            assert rel(d.get(out, (n, pad8(width)))[:, :width], want[at:at + n]) < 1e-6
            at += n


# ---- products --------------------------------------------------------------------------------

@pytest.mark.parametrize("rows,cols,batch", [(40, 24, 1), (333, 76, 3), (128, 264, 70), (96, 4096, 5)])
def test_squared_relu_behind_a_product(gpu, rows, cols, batch):
    rng = np.random.default_rng(rows)
    w, x = weights(rng, rows, cols), weights(rng, batch, cols, scale=1.0)
    want = npl.relu_squared(x.astype(np.float64) @ w.T.astype(np.float64))
    padded = np.zeros((batch, pad8(cols)), np.float32)
    padded[:, :cols] = x
    with Dev(gpu) as d:
        out = d.zeros(batch * rows * 4)
        d.call("lv_gemv_bf16", out, rows, d.bf16(w), rows, pad8(cols), cols, d.f32(padded), pad8(cols), batch, 1.0, 1)
        assert rel(d.get(out, (batch, rows)), want) < 1e-6
        d.call("lv_gemm_bf16", out, pkg.TYPE_F32, rows, d.bf16(w), rows, pad8(cols), cols, d.bf16(x), pad8(cols), batch, 1.0, 1)
        assert rel(d.get(out, (batch, rows)), want) < 2e-5


@pytest.mark.parametrize("window,pos,batch", [(0, 0, 5), (0, 130, 2), (1, 40, 3), (20, 7, 9), (20, 19, 2), (20, 20, 2), (64, 100, 70), (130, 300, 200), (600, 300, 12)])
def test_products_of_the_rows_in_a_window(gpu, window, pos, batch):
    rng = np.random.default_rng(window + pos)
    rows, cols, total = 144, 72, 512
    w, x = weights(rng, rows, cols), weights(rng, total, cols, scale=1.0)
    first = max(0, pos + 1 - window) if window else 0
    n = pos + batch - first
    bound = min(total, window + batch - 1 if window else total)
    with Dev(gpu) as d:
        out = d.up(np.full(bound * rows, -7.0, np.float32))
        d.call("lv_gemm_bf16_window", out, pkg.TYPE_F32, rows, d.bf16(w), rows, pad8(cols), cols, d.bf16(x), pad8(cols), total, d.u32([pos] * 4), batch, window, bound)
        got = d.get(out, (bound, rows))
    assert rel(got[:n], x[first:pos + batch].astype(np.float64) @ w.T.astype(np.float64)) < 2e-5
    assert (got[n:] == -7.0).all()


# ---- rotation --------------------------------------------------------------------------------

@pytest.mark.parametrize("pos,batch", [(0, 1), (0, 70), (1000003, 3)])
def test_rotary_table(gpu, pos, batch):
    parts = [npl.yarn(16, 2e5, {"factor": 3.0, "original": 100, "fast": 16.0, "slow": 1.0}), npl.yarn(6, 500.0)]
    freqs, mults = np.concatenate([p[0] for p in parts]), np.concatenate([np.full(len(p[0]), p[1]) for p in parts]).astype(np.float32)
    with Dev(gpu) as d:
        out = d.zeros(batch * len(freqs) * 8)
        d.call("lv_rotary_table", out, d.up(freqs), d.f32(mults), len(freqs), d.u32([pos] * 4), batch)
        got = d.get(out, (batch, len(freqs), 2))
    a = (pos + np.arange(batch))[:, None] * freqs
    assert np.abs(got - np.stack([np.cos(a), np.sin(a)], axis=-1) * mults[:, None]).max() < 3e-7


# ---- attention over a latent cache ------------------------------------------------------------

ABSORBED, EXPANDED = 1, 2


class Latent:
    """One sequence through lv_latent_attention in portions; `reader` instances use another one's cache."""

    def __init__(self, d, rng, H, dim, rot, vdim, rank, window, rows, f32, scale=None, owner=None, pairs=None, sink=True):
        self.d, self.H, self.dim, self.rot, self.vdim, self.rank, self.window, self.rows, self.f32 = d, H, dim, rot, vdim, rank, window, rows, f32
        self.scale, self.owner = scale or 1.5 * (dim + rot) ** -0.5, owner
        self.uk, self.uv = weights(rng, H * dim, rank), weights(rng, H * vdim, rank)
        self.sink = (rng.standard_normal(H) * 1.5).astype(np.float32) if sink else None
        self.norm = (1 + 0.4 * rng.standard_normal(rank)).astype(np.float32)
        self.pairs = rot // 2 if pairs is None else pairs
        self.freqs, self.mult = npl.yarn(2 * self.pairs, 300.0, {"factor": 2.0, "original": 50, "fast": 6.0, "slow": 0.5}) if self.pairs else (np.zeros(0), 1.0)
        self.w = d.bf16(np.concatenate([self.uk, self.uv]))
        self.dnorm, self.dsink = d.f32(self.norm), d.f32(self.sink) if sink else None
        self.cache = owner.cache if owner else nans(d, rows * (pad8(rank) + pad8(rot)) * (4 if f32 else 2))      # only written rows may count

    def draw(self, rng, T):
        return rng.standard_normal((T, self.H * (self.dim + self.rot))).astype(np.float32), rng.standard_normal((T, self.rank + self.rot)).astype(np.float32)

    def run(self, q, dkv, at, form=0, bf16_out=False):
        d, n = self.d, q.shape[0]
        a = (at + np.arange(n))[:, None] * self.freqs
        angles = d.f32(np.stack([np.cos(a), np.sin(a)], axis=-1) * self.mult) if self.pairs else d.zeros(16)
        ld = pad8(self.H * self.vdim)
        out = nans(d, n * ld * 4)
        args = pkg.LatentArgs(q=d.f32(q).value, q_ld=q.shape[1], dkv=d.f32(dkv).value if self.owner is None else None, dkv_ld=dkv.shape[1], heads=self.H, dim=self.dim, rot=self.rot,
                              vdim=self.vdim, kv_rank=self.rank, scale=self.scale, eps=EPS, kv_norm=self.dnorm.value, angles=angles.value, angle_ld=2 * self.pairs,
                              angle_pairs=self.pairs, w=self.w.value, w_ld=pad8(self.rank), sink=self.dsink.value if self.dsink else None, window=self.window,
                              cache=self.cache.value, cache_type=pkg.TYPE_F32 if self.f32 else pkg.TYPE_BF16, ctx_rows=self.rows, pos=d.u32([at] * 4).value, out=out.value,
                              out_type=pkg.TYPE_BF16 if bf16_out else pkg.TYPE_F32, out_ld=ld, form=form)
        nbytes = d.gpu.lib.lv_latent_scratch_bytes(d.gpu.handle, C.byref(args), n, self.rows)
        d.call("lv_latent_attention", C.byref(args), nans(d, nbytes), nbytes, n, self.rows)
        return d.get(out, (n, ld), bf16_out)[:, :self.H * self.vdim]

    def plain(self, q, dkv):
        owner = self.owner or self
        T, pos = q.shape[0], np.arange(q.shape[0]).astype(np.float64)
        q = q.astype(np.float64).reshape(T, self.H, self.dim + self.rot)
        turn = lambda v: npl.rotate(v.astype(np.float64), pos, self.freqs, self.mult)
        q = np.concatenate([q[..., :self.dim], turn(q[..., self.dim:])], axis=-1)
        c = sp.norm_plain(dkv[:, :self.rank].astype(np.float64), owner.norm.astype(np.float64), EPS)
        sink = self.sink.astype(np.float64) if self.sink is not None else np.full(self.H, -1e30)
        return npl.latent_attention(q, c, turn(dkv[:, self.rank:]), self.uk.astype(np.float64), self.uv.astype(np.float64), sink, self.scale, self.window or T + 1)


CUTS = [[1] * 40, [150], [100, 1, 1, 30, 2, 3, 1], [2] * 33]


@pytest.mark.parametrize("H,dim,rot,vdim,rank,window", [
    (3, 24, 8, 40, 48, 20), (1, 16, 2, 8, 8, 1), (9, 64, 16, 48, 136, 72), (8, 128, 64, 128, 512, 65), (5, 20, 6, 12, 36, 31), (2, 13, 4, 9, 20, 2), (4, 32, 32, 200, 96, 0),
    (17, 40, 24, 16, 264, 64), (2, 256, 0, 64, 72, 100), (2, 128, 100, 256, 1000, 33), (3, 72, 10, 24, 640, 200)])
@pytest.mark.parametrize("f32", [True, False])
def test_latent_attention_in_portions(gpu, H, dim, rot, vdim, rank, window, f32):
    rng = np.random.default_rng(H * dim + rank)
    for cuts in CUTS:
        with Dev(gpu) as d:
            at = Latent(d, rng, H, dim, rot, vdim, rank, window, 256, f32)
            q, dkv = at.draw(rng, sum(cuts))
            want, done = at.plain(q, dkv), 0
            for n in cuts:
                got = at.run(q[done:done + n], dkv[done:done + n], done, bf16_out=not f32 and n > 1)
                assert rel(got, want[done:done + n]) < (3e-6 if f32 else 1.2e-2), (done, n)
                done += n


@pytest.mark.parametrize("form", [ABSORBED, EXPANDED])
@pytest.mark.parametrize("H,dim,rot,vdim,rank,window", [(3, 24, 8, 40, 48, 20), (6, 64, 16, 48, 128, 130), (2, 128, 64, 128, 512, 0)])
def test_both_forms_take_any_portion(gpu, form, H, dim, rot, vdim, rank, window):
    rng = np.random.default_rng(form)
    cuts = [2, 3, 5, 128, 2, 129, 4, 3] if form == EXPANDED else [1, 2, 3, 1, 128, 1, 1, 129, 4, 3]
    with Dev(gpu) as d:
        at = Latent(d, rng, H, dim, rot, vdim, rank, window, 320, False)
        q, dkv = at.draw(rng, sum(cuts))
        want, done = at.plain(q, dkv), 0
        for n in cuts:
            assert rel(at.run(q[done:done + n], dkv[done:done + n], done, form), want[done:done + n]) < 1.2e-2, (done, n)
            done += n


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("window,form", [(0, 0), (1500, 0), (0, ABSORBED), (1100, ABSORBED)])
@pytest.mark.parametrize("H,rank", [(3, 40), (11, 520), (35, 72)])
def test_decoding_far_into_a_sequence(gpu, f32, window, form, H, rank):
    """More visible rows than shared memory holds at a time, and a step's own row in any place of a chunk."""
    rng = np.random.default_rng(H)
    T, steps = 2100, 34
    with Dev(gpu) as d:
        at = Latent(d, rng, H, 16, 8, 16, rank, window, 2200, f32)
        q, dkv = at.draw(rng, T)
        for first in range(0, T - steps, 512):
            last = min(first + 512, T - steps)
            at.run(q[first:last], dkv[first:last], first)
        got = np.concatenate([at.run(q[i:i + 1], dkv[i:i + 1], i, form) for i in range(T - steps, T)])
        # plain, for the decoded positions only
        pos = np.arange(T).astype(np.float64)
        c = sp.norm_plain(dkv[:, :rank].astype(np.float64), at.norm.astype(np.float64), EPS)
        kr = npl.rotate(dkv[:, rank:].astype(np.float64), pos, at.freqs, at.mult)
        qq = q[T - steps:].astype(np.float64).reshape(steps, H, 24)
        qr = npl.rotate(qq[..., 16:], pos[T - steps:], at.freqs, at.mult)
        k, v = (c @ at.uk.T.astype(np.float64)).reshape(T, H, 16), (c @ at.uv.T.astype(np.float64)).reshape(T, H, 16)
        s = (np.einsum("ihd,jhd->hij", qq[..., :16], k) + np.einsum("ihd,jd->hij", qr, kr)) * at.scale
        p = npl.sink_weights(s, npl.window_mask(T, window or T + 1)[T - steps:], at.sink.astype(np.float64))
        want = np.einsum("hij,jhd->ihd", p, v).reshape(steps, -1)
    assert rel(got, want) < (5e-6 if f32 else 1.2e-2)


@pytest.mark.parametrize("f32", [True, False])
def test_layers_that_read_another_layers_cache(gpu, f32):
    """Other heads, value sizes, windows and sinks over the same rows."""
    rng = np.random.default_rng(5)
    with Dev(gpu) as d:
        at = Latent(d, rng, 3, 24, 8, 40, 48, 20, 256, f32)
        reader = Latent(d, rng, 5, 16, 8, 24, 48, 75, 256, f32, owner=at)
        q, dkv = at.draw(rng, 120)
        q2, _ = reader.draw(rng, 120)
        want, want2 = at.plain(q, dkv), reader.plain(q2, dkv)
        done = 0
        for n in (60, 1, 1, 2, 50, 1, 5):
            assert rel(at.run(q[done:done + n], dkv[done:done + n], done), want[done:done + n]) < (3e-6 if f32 else 1.2e-2)
            assert rel(reader.run(q2[done:done + n], dkv[done:done + n], done), want2[done:done + n]) < (3e-6 if f32 else 1.2e-2)
            done += n


@pytest.mark.parametrize("f32,n,form", [(True, 1, 0), (True, 2, 0), (True, 37, 0), (False, 1, 0), (False, 2, ABSORBED), (False, 2, EXPANDED), (False, 37, ABSORBED),
                                        (False, 37, EXPANDED), (False, 150, EXPANDED)])
@pytest.mark.parametrize("window", [33, 64, 96])
def test_the_edge_of_the_window(gpu, f32, n, form, window):
    """One key stands out for every query: it decides the output just inside the window and is gone just outside."""
    rng = np.random.default_rng(window)
    H, dim, rot, vdim, rank, T = 3, 32, 8, 24, 64, 330
    with Dev(gpu) as d:
        at = Latent(d, rng, H, dim, rot, vdim, rank, window, 384, f32, scale=1.0, pairs=0)            # no rotation: the key stands out at any distance
        q, dkv = at.draw(rng, T)
        q *= 0.05
        mark = rng.standard_normal(rot)
        dkv[:, rank:] *= 0.05
        q.reshape(T, H, dim + rot)[:, :, dim:] = mark * 3
        for target in {T - n, T - 1, T - n // 2 - 1}:            # queries whose edge is looked at
            for distance in (window - 2, window - 1, window, window + 1):
                k = dkv.copy()
                k[target - distance, rank:] = mark * 3
                want = at.plain(q, k)
                at.run(q[:T - n], k[:T - n], 0)
                got = at.run(q[T - n:], k[T - n:], T - n, form)
                assert rel(got, want[T - n:]) < (1e-5 if f32 else 1.5e-2), (target, distance)
                only = (at.uv.astype(np.float64) @ sp.norm_plain(k[target - distance:target - distance + 1, :rank].astype(np.float64), at.norm.astype(np.float64), EPS)[0])
                seen = np.corrcoef(got[target - (T - n)], only)[0, 1] > 0.98
                assert seen == (distance < window), (target, distance)


@pytest.mark.parametrize("f32", [True, False])
def test_a_single_far_latent_key_is_found(gpu, f32):
    rng = np.random.default_rng(11)
    H, dim, rot, vdim, rank, T = 4, 64, 16, 48, 96, 530
    for window in (0, 529):
        for far in (1, 31, 32, 63, 64, 65, 127, 128, 300, 511, 512, 527):
            with Dev(gpu) as d:
                at = Latent(d, rng, H, dim, rot, vdim, rank, window, 640, f32, scale=1.0)
                q, dkv = at.draw(rng, T)
                q[-2:] *= 0.02
                c = sp.norm_plain(dkv[far:far + 1, :rank].astype(np.float64), at.norm.astype(np.float64), EPS)[0]
                q[-2:].reshape(2, H, dim + rot)[:, :, :dim] = 0.6 * (at.uk @ c).reshape(H, dim)
                want = at.plain(q, dkv)
                at.run(q[:T - 2], dkv[:T - 2], 0)
                two = at.run(q[T - 2:], dkv[T - 2:], T - 2, 0 if f32 else EXPANDED)
                one = at.run(q[T - 1:], dkv[T - 1:], T - 1)
                assert rel(two, want[-2:]) < (1e-5 if f32 else 1.5e-2) and rel(one, want[-1:]) < (1e-5 if f32 else 1.5e-2), (window, far)
                assert np.corrcoef(one[0], at.uv @ c)[0, 1] > 0.98


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("sinks", [[30.0, -30.0, 0.0], [3.0, 5.0, -80.0]])
def test_sinks_of_any_height(gpu, f32, sinks):
    rng = np.random.default_rng(2)
    with Dev(gpu) as d:
        at = Latent(d, rng, 3, 24, 8, 16, 40, 12, 128, f32)
        at.sink = np.array(sinks, np.float32)
        at.dsink = d.f32(at.sink)
        q, dkv = at.draw(rng, 90)
        want = at.plain(q, dkv).reshape(90, 3, 16)
        whole = at.run(q, dkv, 0).reshape(90, 3, 16)
        one = np.concatenate([at.run(q[i:i + 1], dkv[i:i + 1], i) for i in range(90)]).reshape(90, 3, 16)
        for h in range(3):                                       # per head: a large sink leaves very little
            assert rel(whole[:, h], want[:, h]) < (5e-6 if f32 else 1.5e-2) and rel(one[:, h], want[:, h]) < (5e-6 if f32 else 1.5e-2)
        at2 = Latent(d, rng, 3, 24, 8, 16, 40, 12, 128, f32, sink=False)
        first = at2.run(q[:1], dkv[:1], 0)                        # without a sink the first token is its own value
        assert rel(first, at2.plain(q[:1], dkv[:1])) < (1e-6 if f32 else 1e-2)


def test_positions_outside_the_latent_cache_are_refused_on_the_device(gpu):
    rng = np.random.default_rng(1)
    for n in (1, 2, 6):
        with Dev(gpu) as d:
            at = Latent(d, rng, 2, 16, 4, 16, 24, 10, 128, False)
            q, dkv = at.draw(rng, n)
            with pytest.raises(pkg.LvError) as e:
                at.run(q, dkv, 128)
            assert e.value.code == pkg.LV_ERR_DEVICE_WAIT


# ---- state space -------------------------------------------------------------------------------

class StateSpace:
    def __init__(self, d, rng, H, P, N, G, taps, parts, A_mean=-1.5, dt_mean=-1.0):
        self.d, self.H, self.P, self.N, self.G, self.taps, self.parts = d, H, P, N, G, taps, parts
        self.inner, self.channels = H * P, H * P + 2 * G * N
        f = lambda *s, mean=0.0, spread=0.4: (mean + spread * rng.standard_normal(s)).astype(np.float32)
        self.conv, self.conv_b, self.D, self.norm = f(self.channels, taps, spread=0.6), f(self.channels), f(H), f(self.inner, mean=1.0)
        self.A_log, self.dt_bias = f(H, mean=A_mean, spread=1.5), f(H, mean=dt_mean, spread=1.0)
        self.dev = [d.f32(np.ascontiguousarray(v)) for v in (self.conv.T, self.conv_b, self.dt_bias, self.A_log, self.D, self.norm)]
        self.history, self.S = nans(d, taps * self.channels * 4), nans(d, H * P * d.gpu.lib.lv_ssm_state_rows(N) * 4)      # no clearing needed

    def draw(self, rng, T):
        return rng.standard_normal((T, 2 * self.inner + 2 * self.G * self.N + self.H)).astype(np.float32)

    def run(self, raw, at, bf16=False, form=0):
        d, n = self.d, raw.shape[0]
        ld = pad8(self.inner)
        out = nans(d, n * ld * 4)
        conv, conv_b, dt_bias, A_log, D, norm = self.dev
        a = pkg.SsmArgs(raw=d.f32(raw).value, raw_ld=raw.shape[1], heads=self.H, vdim=self.P, state=self.N, groups=self.G, taps=self.taps, conv_w=conv.value, conv_b=conv_b.value,
                        dt_bias=dt_bias.value, A_log=A_log.value, D=D.value, norm_w=norm.value, norm_groups=self.parts, eps=EPS, history=self.history.value, S=self.S.value,
                        pos=d.u32([at] * 4).value, out=out.value, out_type=pkg.TYPE_BF16 if bf16 else pkg.TYPE_F32, out_ld=ld, form=form)
        nbytes = d.gpu.lib.lv_ssm_scratch_bytes(C.byref(a), n)
        d.call("lv_ssm", C.byref(a), nans(d, nbytes), nbytes, n)
        return d.get(out, (n, ld), bf16)[:, :self.inner]

    def plain(self, raw, rounded=False):
        """rounded: x, B and C in bfloat16"""
        T = raw.shape[0]
        z, xbc, dt = np.split(raw.astype(np.float64), [self.inner, self.inner + self.channels], axis=1)
        xbc = sp.silu(sp.causal_conv(xbc, self.conv.astype(np.float64)) + self.conv_b)
        if rounded:
            xbc = sp.bf16_round(xbc.astype(np.float32)).astype(np.float64)
        x, B, K = np.split(xbc, [self.inner, self.inner + self.G * self.N], axis=1)
        y = npl.state_space(x.reshape(T, self.H, self.P), B.reshape(T, self.G, self.N), K.reshape(T, self.G, self.N), npl.softplus(dt + self.dt_bias),
                            self.A_log.astype(np.float64), self.D.astype(np.float64))
        return npl.gated_group_norm(y.reshape(T, self.inner), z, self.norm.astype(np.float64), self.parts, EPS)


SIZES = [(6, 20, 24, 2, 3, 3), (4, 32, 16, 4, 5, 1), (3, 40, 130, 1, 2, 1), (8, 64, 128, 2, 4, 8), (5, 9, 11, 5, 7, 3), (2, 300, 8, 1, 1, 2), (10, 12, 64, 5, 16, 5), (1, 7, 256, 1, 4, 1)]


@pytest.mark.parametrize("H,P,N,G,taps,parts", SIZES)
@pytest.mark.parametrize("cuts", [[1] * 40, [140], [33, 1, 1, 2, 31, 64, 3, 1, 1, 2], [2] * 20, [32, 32, 1], [640, 1, 131]])
def test_state_space_in_portions(gpu, H, P, N, G, taps, parts, cuts):
    rng = np.random.default_rng(H * P + N)
    with Dev(gpu) as d:
        s = StateSpace(d, rng, H, P, N, G, taps, parts)
        raw = s.draw(rng, sum(cuts))
        want, at = s.plain(raw), 0
        for n in cuts:
            assert rel(s.run(raw[at:at + n], at), want[at:at + n]) < 5e-6, (at, n)
            at += n


TENSOR = 2


@pytest.mark.parametrize("H,P,N,G,taps,parts", [(4, 32, 16, 4, 5, 1), (3, 40, 130, 1, 2, 1), (8, 64, 128, 2, 4, 8), (6, 8, 11, 3, 7, 3), (2, 304, 8, 1, 1, 2), (10, 16, 64, 5, 16, 5),
                                                (1, 24, 256, 1, 4, 1), (5, 48, 33, 1, 3, 1), (80, 64, 16, 2, 2, 4), (76, 40, 72, 1, 3, 1)])
@pytest.mark.parametrize("cuts", [[140], [33, 2, 31, 64, 3, 2], [2] * 20, [64, 64, 65], [63, 700]])
def test_chunks_of_tokens_as_matrix_products(gpu, H, P, N, G, taps, parts, cuts):
    """Everything but x, B and C is as exact as in f32."""
    rng = np.random.default_rng(H * P + N)
    with Dev(gpu) as d:
        s = StateSpace(d, rng, H, P, N, G, taps, parts)
        raw = s.draw(rng, sum(cuts))
        want, at = s.plain(raw, rounded=True), 0
        for n in cuts:
            far = rel(s.run(raw[at:at + n], at, form=TENSOR), want[at:at + n])
            assert far < 4e-4, (at, n)                            # (a convolution's output at the middle between two bfloat16 numbers rounds either way)
            at += n


@pytest.mark.parametrize("A_mean,dt_mean", [(-6.0, -5.0), (-9.0, 0.5), (2.0, 3.0), (5.0, 6.0), (1.0, -1.0)])
def test_matrix_products_and_scan_take_turns(gpu, A_mean, dt_mean):
    """Weak to complete decays; the state that one form leaves is what the other (and a single token) continues from."""
    rng = np.random.default_rng(4)
    with Dev(gpu) as d:
        s = StateSpace(d, rng, 6, 24, 32, 2, 4, 2, A_mean, dt_mean)
        raw = s.draw(rng, 400)
        raw[:, -6:] *= 3
        want, at = s.plain(raw), 0
        for n, form in ((100, TENSOR), (70, 1), (1, 0), (129, TENSOR), (1, 0), (99, TENSOR)):
            assert rel(s.run(raw[at:at + n], at, form=form), want[at:at + n]) < 1e-2, (at, n)
            at += n


@pytest.mark.parametrize("A_mean,dt_mean", [(-6.0, -5.0), (2.0, 3.0), (5.0, 6.0), (1.0, -1.0)])
def test_decays_from_almost_none_to_complete(gpu, A_mean, dt_mean):
    """Logarithms of decays from -1e-5 to far below what f32 can represent, mixed within a chunk by dt."""
    rng = np.random.default_rng(4)
    with Dev(gpu) as d:
        s = StateSpace(d, rng, 6, 24, 32, 2, 4, 2, A_mean, dt_mean)
        raw = s.draw(rng, 300)
        raw[:, -6:] *= 3
        want = s.plain(raw)
        assert rel(s.run(raw[:280], 0), want[:280]) < 1e-5
        got = np.concatenate([s.run(raw[i:i + 1], i) for i in range(280, 300)])
        assert rel(got, want[280:]) < 1e-5


def test_a_token_far_back_is_remembered(gpu):
    """Slow decays: the state written by one early token decides what is read 400 tokens later, decoded or not."""
    rng = np.random.default_rng(9)
    with Dev(gpu) as d:
        s = StateSpace(d, rng, 2, 16, 24, 1, 2, 1, A_mean=-9.0, dt_mean=0.5)
        raw = s.draw(rng, 420)
        raw[5:, s.inner:2 * s.inner] = 0                          # after the first tokens nothing is written
        s.conv_b[:] = 0
        s.dev[1] = d.f32(s.conv_b)
        want = s.plain(raw)
        whole = s.run(raw[:400], 0)
        assert rel(whole[390:], want[390:400]) < 1e-5
        one = np.concatenate([s.run(raw[i:i + 1], i) for i in range(400, 420)])
        assert rel(one, want[400:]) < 1e-5 and np.abs(want[400:]).max() > 0.1


def test_state_space_output_in_bfloat16(gpu):
    rng = np.random.default_rng(4)
    with Dev(gpu) as d:
        s = StateSpace(d, rng, 4, 24, 16, 2, 4, 2)
        raw = s.draw(rng, 50)
        assert rel(s.run(raw, 0, bf16=True), s.plain(raw)) < 4e-3


def test_bad_arguments_are_refused(gpu):
    lib, h, bad = gpu.lib, gpu.handle, pkg.LV_ERR_BAD_ARGUMENTS
    with Dev(gpu) as d:
        b = d.zeros(1 << 16)
        v = b.value
        assert lib.lv_gemv_bf16(h, b, 16, b, 8, 16, 16, b, 16, 1, 1.0, 9) == bad                       # unknown activation
        good = dict(q=v, q_ld=64, dkv=v, dkv_ld=64, heads=2, dim=16, rot=4, vdim=16, kv_rank=24, scale=1.0, eps=EPS, kv_norm=v, angles=v, angle_ld=4, angle_pairs=2, w=v, w_ld=24,
                    sink=v, window=5, cache=v, cache_type=pkg.TYPE_F32, ctx_rows=64, pos=v, out=v, out_type=pkg.TYPE_F32, out_ld=32, form=0)
        for change in (dict(q_ld=30), dict(w_ld=20), dict(angle_pairs=3), dict(kv_rank=1025, w_ld=1032), dict(form=EXPANDED), dict(out=None), dict(kv_norm=None)):
            a = pkg.LatentArgs(**{**good, **change})
            assert lib.lv_latent_attention(h, C.byref(a), b, 1 << 16, 2, 64) == bad, change
        assert lib.lv_latent_attention(h, C.byref(pkg.LatentArgs(**good)), b, 64, 1, 64) == bad           # scratch too small
        good = dict(raw=v, raw_ld=400, heads=4, vdim=8, state=16, groups=2, taps=4, conv_w=v, conv_b=v, dt_bias=v, A_log=v, D=v, norm_w=v, norm_groups=2, eps=EPS, history=v, S=v,
                    pos=v, out=v, out_type=pkg.TYPE_F32, out_ld=32)
        for change in (dict(groups=3), dict(norm_groups=5), dict(state=257), dict(taps=17), dict(raw_ld=20), dict(out_ld=8)):
            assert lib.lv_ssm(h, C.byref(pkg.SsmArgs(**{**good, **change})), b, 1 << 16, 1) == bad, change
