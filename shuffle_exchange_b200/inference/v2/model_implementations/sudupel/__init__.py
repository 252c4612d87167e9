from .policy import SudupelPolicy  # noqa: F401
