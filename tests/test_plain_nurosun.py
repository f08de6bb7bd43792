"""The restatement the GPU tests of Nurosun trust, checked against properties of its mechanisms."""
import numpy as np

import _plain_nurosun as plain
from _nurosun_models import config, dense, latent, moe, tokens, weights


def test_no_lookahead():
    cfg = config([latent(mlp=dense(20)), latent(source=0, mlp=moe())])
    w, t = weights(cfg, 1), None
    t = tokens(cfg, 30, 2)
    assert np.abs(plain.forward(cfg, w, t[:12]) - plain.forward(cfg, w, t)[:12]).max() < 1e-10


def test_rotation_depends_on_distance_only():
    rng = np.random.default_rng(1)
    q, k = rng.standard_normal((1, 10)), rng.standard_normal((1, 10))
    dots = [(plain.rotate_half(q, [p + 7], 50.0) @ plain.rotate_half(k, [p], 50.0).T).item() for p in (0, 3, 1000)]
    assert np.ptp(dots) < 1e-10
    assert np.allclose(plain.rotate_half(q, [0], 50.0), q)


def test_norms_and_routing():
    rng = np.random.default_rng(2)
    x = rng.standard_normal((4, 31)) * 5 + 3
    y = plain.layer_norm(x, np.ones(31), 0.0)
    assert np.allclose(y.mean(-1), 0) and np.allclose((y ** 2).mean(-1), 1)
    chosen, weight = plain.route(x, rng.standard_normal((9, 31)), rng.standard_normal(9), 4)
    assert np.allclose(weight.sum(-1), 1) and (np.diff(weight) <= 0).all() and all(len(set(r)) == 4 for r in chosen.tolist())


def test_absorbed_scores_are_the_same():
    """q . (U c) = (U^T q) . c: what the product's decode path computes."""
    rng = np.random.default_rng(3)
    u, c, q = rng.standard_normal((6, 11)), rng.standard_normal((5, 11)), rng.standard_normal(6)
    assert np.allclose((c @ u.T) @ q, c @ (u.T @ q))
