"""Architecture families, one module each; importing this package registers them."""

from mlx_omnia_b200.architectures import bobarax, dolutar, fokalorn, gisudra, muse_glimmer, narezen, rinirax  # noqa: F401
